// attention_talking.cu -- softmax attention whose heads exchange their scores before the softmax, over the paged cache, for ragged steps (portions of
// prompts beside single decoded tokens in one launch).  Per query i of a sequence and visible key j:
//     s[h, j] = scale q[h] . k_j[kv(h)],   s'[h, j] = sum_g talk[h, g] s[g, j],   p = exp(s') / (one_sink + sum_j exp(s')),   o[h] = sum_j p[h, j] v_j[kv(h)]
// kv(h) = floor(h / (H / G)); one_sink = 1 is a key without a value whose score is 0.  Key j is visible iff j <= i, j / chunk == i / chunk (chunk > 0)
// and i - j < window (window > 0), all counted in sequence positions.  With cos / sin tables [max_pos, dv/2] the cached values have been turned by their
// position, and o[h] is turned back by the query's (pair m with m + dv/2 by minus the table's angle) before it is written.
//
// Because a query's softmax needs the raw scores of ALL heads, the unit of work is a query (or a tile of queries) with all its heads:
//   talking_rows_kernel     a block per (row, run of keys), f32 arithmetic, any sizes, f32 or bf16 cache: scores (a warp per kv head and 32 keys, four lanes
//                           share a key's row in 16-byte pieces), mixing and online softmax (a warp per head, a lane per key), values (a warp per run of
//                           heads, lanes across the columns).  Few rows: the keys of a row are cut into runs and talking_merge_kernel joins them.
//   talking_decode_kernel   the same for few rows over a 16-bit cache, on mma.sync: every head gets a mixed query as long as a cache row.
//   talking_prefill_kernel  portions of prompts in 16 bits: a block per 8 query rows with ALL heads, mma.sync m16n8k16 with keys (or value columns) on the
//                           16-row side and queries on the 8-column side, so that 32 heads' accumulators of 128 value columns fit the register file.  A warp
//                           owns H / 16 heads in both products; raw scores meet in shared memory in f32, are mixed there on the tensor
//                           cores as sums of three 16-bit parts (all 24 bits of a score), and every warp reads its heads' mixed scores back in the operand
//                           layout of the second product.  The first product of the
//                           next tile is issued before the mixing of this one (scores double-buffered), so a tile costs one barrier; keys and values
//                           arrive by cp.async while earlier tiles are worked on.
#include <cuda.h>

#include "common.cuh"

namespace b200 {
namespace {

struct TalkArgs {
    const float* q;                              // [T, H dk]
    const void* kc; const void* vc;              // [nb, bs, G, dk], [nb, bs, G, dv]
    const int32_t* block_tables; int table_width;
    const int32_t* token_seq; const int32_t* positions;
    const float* talk;                           // [H, H] or null
    const float* cos_t; const float* sin_t;      // [max_pos, dv/2] or null
    void* out;                                   // [T, H dv]
    float* part;                                 // splits > 1: [T, splits, H, dv + 2]: unnormalised sum, maximum, denominator
    int H, G, dk, dv, bs;
    float scale;
    int chunk, window, one_sink, splits, tile, qpitch, bs_shift;
};

// cache row of a position (shift >= 0: the block size is 1 << shift, otherwise it is divided by)
__device__ __forceinline__ int cache_row(const int32_t* table, int j, int bs, int shift) {
    const int b = shift >= 0 ? j >> shift : j / bs;
    return table[b] * bs + (j - b * bs);
}
__device__ __forceinline__ int first_visible(int pos, int chunk, int window) {
    int lo = chunk > 0 ? (pos / chunk) * chunk : 0;
    if (window > 0 && pos - window + 1 > lo) lo = pos - window + 1;
    return lo;
}

template <typename TC> struct Piece;             // a 16-byte piece of a cached row as floats, and four neighbouring entries of one
template <> struct Piece<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void open(const uint4& r, float (&v)[4]) {
        v[0] = __uint_as_float(r.x); v[1] = __uint_as_float(r.y); v[2] = __uint_as_float(r.z); v[3] = __uint_as_float(r.w);
    }
    typedef float4 Four;
    static __device__ __forceinline__ float4 four(const float4& w) { return w; }
};
template <> struct Piece<__nv_bfloat16> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void open(const uint4& r, float (&v)[8]) {
        const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) { v[2 * i] = __uint_as_float(w[i] << 16); v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u); }
    }
    typedef uint2 Four;
    static __device__ __forceinline__ float4 four(const uint2& w) {
        return make_float4(__uint_as_float(w.x << 16), __uint_as_float(w.x & 0xffff0000u), __uint_as_float(w.y << 16), __uint_as_float(w.y & 0xffff0000u));
    }
};

// kHW: heads a warp accumulates values for, kC: groups of four value columns per lane (columns 4 lane + 128 c and the next three)
template <typename TC, typename TOut, int kHW, int kC>
__global__ void __launch_bounds__(256, kHW * kC <= 2 ? 2 : 1)
talking_rows_kernel(const TalkArgs A) {
    pdl_wait();
    pdl_trigger();
    constexpr int N = Piece<TC>::N;
    extern __shared__ __align__(16) float sm[];
    const int H = A.H, G = A.G, dk = A.dk, dv = A.dv, KT = A.tile, group = H / G, qp = A.qpitch;
    float* qs = sm;                              // [H][qp] scaled queries, zeros past dk
    float* S = qs + H * qp;                      // [H][KT] raw scores
    float* P = S + H * KT;                       // [H][KT] weights
    const int pool = max(2 * H * KT, max(8, H) * dv);
    float* ms = S + ((pool + 3) & ~3);           // [H] running maximum, [H] denominator, [H] correction of this tile
    float* ls = ms + H; float* cs = ls + H;
    int64_t* ph = reinterpret_cast<int64_t*>(ms + ((3 * H + 3) & ~3));       // [2][KT] cache rows of the tile's keys
    float* tk = reinterpret_cast<float*>(ph + 2 * KT);                       // [H][H]
    const int t = blockIdx.x, split = blockIdx.y;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int pos = A.positions[t];
    const int lo = first_visible(pos, A.chunk, A.window);
    const int per = ((pos - lo + A.splits) / A.splits + 31) & ~31;
    const int jb = lo + split * per, je = min(pos + 1, jb + per);
    const int32_t* table = A.block_tables + (int64_t)A.token_seq[t] * A.table_width;
    const TC* kc = static_cast<const TC*>(A.kc);
    const TC* vc = static_cast<const TC*>(A.vc);
    for (int i = threadIdx.x; i < H * qp; i += 256) {
        const int h = i / qp, d = i - h * qp;
        qs[i] = d < dk ? A.q[((int64_t)t * H + h) * dk + d] * A.scale : 0.f;
    }
    if (A.talk) for (int i = threadIdx.x; i < H * H; i += 256) tk[i] = A.talk[i];
    for (int h = threadIdx.x; h < H; h += 256) {
        const bool sink = A.one_sink && split == 0;                          // a key of score 0 without a value, counted by the first run
        ms[h] = sink ? 0.f : -INFINITY;
        ls[h] = sink ? 1.f : 0.f;
    }
    auto place = [&](int j0, int buf) {          // keys past the run's end stand for its first one (their weight is 0, what they read is finite)
        for (int i = threadIdx.x; i < KT; i += 256) {
            const int j = j0 + i < je ? j0 + i : jb;
            ph[buf * KT + i] = cache_row(table, j, A.bs, A.bs_shift);
        }
    };
    if (jb < je) place(jb, 0);
    // value heads of this warp; with fewer than eight heads the warps share a head's keys
    const int slices = H < 8 ? 8 / H : 1;
    const int h0 = H < 8 ? warp % H : warp * kHW, slice = H < 8 ? warp / H : 0;
    const bool has_values = slice < slices && h0 < H;
    int kvh[kHW];                                // their kv heads
#pragma unroll
    for (int a = 0; a < kHW; ++a) kvh[a] = min(h0 + a, H - 1) / group;
    float4 acc[kHW][kC];
#pragma unroll
    for (int a = 0; a < kHW; ++a)
#pragma unroll
        for (int c = 0; c < kC; ++c) acc[a][c] = make_float4(0.f, 0.f, 0.f, 0.f);
    const bool whole = dk % N == 0, fours = dv % 4 == 0;               // key rows are whole 16-byte pieces, value rows whole groups of four
    __syncthreads();
    for (int j0 = jb, it = 0; j0 < je; j0 += KT, ++it) {
        const int64_t* pht = ph + (it & 1) * KT;
        // ---- raw scores ---------------------------------------------------------------------------------------------------------------
        const int r = lane >> 2, c4 = lane & 3;
        for (int u = warp; u < G * (KT >> 5); u += 8) {
            const int g = u % G, sub = u / G;
            if (j0 + sub * 32 >= je) continue;
            const TC* kp[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) kp[i] = kc + (pht[sub * 32 + i * 8 + r] * G + g) * dk;
            for (int hb = 0; hb < group; hb += 4) {
                float a[4][4] = {};
                uint4 nx[4];                     // the next pieces travel while these are multiplied
#pragma unroll
                for (int i = 0; i < 4; ++i) nx[i] = whole && c4 * N < dk ? *reinterpret_cast<const uint4*>(kp[i] + c4 * N) : make_uint4(0u, 0u, 0u, 0u);
                for (int d0 = 0; d0 < dk; d0 += 4 * N) {
                    const int d = d0 + c4 * N;
                    float kv[4][N];
                    if (whole) {
#pragma unroll
                        for (int i = 0; i < 4; ++i) Piece<TC>::open(nx[i], kv[i]);
                        if (d0 + 4 * N < dk) {
#pragma unroll
                            for (int i = 0; i < 4; ++i) nx[i] = d + 4 * N < dk ? *reinterpret_cast<const uint4*>(kp[i] + d + 4 * N) : make_uint4(0u, 0u, 0u, 0u);
                        }
                    } else {
#pragma unroll
                        for (int i = 0; i < 4; ++i)
#pragma unroll
                            for (int e = 0; e < N; ++e) kv[i][e] = d + e < dk ? to_f32<TC>(kp[i][d + e]) : 0.f;
                    }
#pragma unroll
                    for (int hh = 0; hh < 4; ++hh) {
                        if (hb + hh >= group) continue;
                        const float4* q4 = reinterpret_cast<const float4*>(qs + (g * group + hb + hh) * qp + d);
#pragma unroll
                        for (int e4 = 0; e4 < N / 4; ++e4) {
                            const float4 qv = q4[e4];
#pragma unroll
                            for (int i = 0; i < 4; ++i)
                                a[hh][i] = fmaf(qv.x, kv[i][e4 * 4], fmaf(qv.y, kv[i][e4 * 4 + 1], fmaf(qv.z, kv[i][e4 * 4 + 2], fmaf(qv.w, kv[i][e4 * 4 + 3], a[hh][i]))));
                        }
                    }
                }
#pragma unroll
                for (int hh = 0; hh < 4; ++hh) {
                    if (hb + hh >= group) continue;
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        a[hh][i] += __shfl_xor_sync(0xffffffffu, a[hh][i], 1);
                        a[hh][i] += __shfl_xor_sync(0xffffffffu, a[hh][i], 2);
                    }
                    const float v = c4 == 0 ? a[hh][0] : c4 == 1 ? a[hh][1] : c4 == 2 ? a[hh][2] : a[hh][3];
                    S[(g * group + hb + hh) * KT + sub * 32 + c4 * 8 + r] = v;
                }
            }
        }
        __syncthreads();
        // ---- mixing and online softmax ------------------------------------------------------------------------------------------------
        const int nsub = (min(KT, je - j0) + 31) >> 5;
        for (int h = warp; h < H; h += 8) {
            float v[4] = {0.f, 0.f, 0.f, 0.f};
            if (A.talk) {
                const float* th = tk + h * H;
                for (int g = 0; g < H; ++g) {
                    const float w = th[g];
#pragma unroll
                    for (int sub = 0; sub < 4; ++sub)
                        if (sub < nsub) v[sub] = fmaf(w, S[g * KT + sub * 32 + lane], v[sub]);
                }
            } else {
#pragma unroll
                for (int sub = 0; sub < 4; ++sub)
                    if (sub < nsub) v[sub] = S[h * KT + sub * 32 + lane];
            }
            float mx = -INFINITY;
#pragma unroll
            for (int sub = 0; sub < 4; ++sub) {
                if (j0 + sub * 32 + lane >= je) v[sub] = -INFINITY;
                mx = fmaxf(mx, v[sub]);
            }
            const float m_old = ms[h], m_new = fmaxf(m_old, warp_max(mx));
            float sum = 0.f;
#pragma unroll
            for (int sub = 0; sub < 4; ++sub) {
                if (sub >= nsub) continue;
                const float p = expf(v[sub] - m_new);                        // exp(-inf) = 0 for the places past the run's end
                P[h * KT + sub * 32 + lane] = p;
                sum += p;
            }
            sum = warp_sum(sum);
            if (lane == 0) {
                const float corr = expf(m_old - m_new);
                cs[h] = corr; ms[h] = m_new;
                ls[h] = fmaf(ls[h], corr, sum);
            }
        }
        if (j0 + KT < je) place(j0 + KT, (it + 1) & 1);
        __syncthreads();
        // ---- values -------------------------------------------------------------------------------------------------------------------
        if (has_values) {
#pragma unroll
            for (int a = 0; a < kHW; ++a) {
                const float corr = h0 + a < H ? cs[h0 + a] : 0.f;
#pragma unroll
                for (int c = 0; c < kC; ++c) { acc[a][c].x *= corr; acc[a][c].y *= corr; acc[a][c].z *= corr; acc[a][c].w *= corr; }
            }
            // eight keys at a time: their rows travel together (rows past the run's end repeat its first one, at weight 0)
            for (int k8 = slice * 8; k8 < nsub * 32; k8 += slices * 8) {
                if (j0 + k8 >= je) break;
                int g_loaded = -1;
                float4 vv[8][kC];
#pragma unroll
                for (int a = 0; a < kHW; ++a) {
                    const int g = kvh[a];
                    if (g != g_loaded) {
                        g_loaded = g;
                        if (fours) {                 // all loads first, clamped instead of guarded: columns past dv are not stored
                            typename Piece<TC>::Four raw[8][kC];
#pragma unroll
                            for (int i = 0; i < 8; ++i)
#pragma unroll
                                for (int c = 0; c < kC; ++c)
                                    raw[i][c] = *reinterpret_cast<const typename Piece<TC>::Four*>(vc + (pht[k8 + i] * G + g) * dv + min(4 * lane + 128 * c, dv - 4));
#pragma unroll
                            for (int i = 0; i < 8; ++i)
#pragma unroll
                                for (int c = 0; c < kC; ++c) vv[i][c] = Piece<TC>::four(raw[i][c]);
                        } else {
#pragma unroll
                            for (int i = 0; i < 8; ++i) {
                                const TC* vp = vc + (pht[k8 + i] * G + g) * dv;
#pragma unroll
                                for (int c = 0; c < kC; ++c) {
                                    const int col = 4 * lane + 128 * c;
                                    vv[i][c] = make_float4(col < dv ? to_f32<TC>(vp[col]) : 0.f, col + 1 < dv ? to_f32<TC>(vp[col + 1]) : 0.f,
                                                           col + 2 < dv ? to_f32<TC>(vp[col + 2]) : 0.f, col + 3 < dv ? to_f32<TC>(vp[col + 3]) : 0.f);
                                }
                            }
                        }
                    }
#pragma unroll
                    for (int i4 = 0; i4 < 2; ++i4) {
                        const float4 p4 = h0 + a < H ? *reinterpret_cast<const float4*>(P + (h0 + a) * KT + k8 + 4 * i4) : make_float4(0.f, 0.f, 0.f, 0.f);
                        const float p[4] = {p4.x, p4.y, p4.z, p4.w};
#pragma unroll
                        for (int i = 0; i < 4; ++i)
#pragma unroll
                            for (int c = 0; c < kC; ++c) {
                                const float4 v = vv[4 * i4 + i][c];
                                acc[a][c].x = fmaf(p[i], v.x, acc[a][c].x); acc[a][c].y = fmaf(p[i], v.y, acc[a][c].y);
                                acc[a][c].z = fmaf(p[i], v.z, acc[a][c].z); acc[a][c].w = fmaf(p[i], v.w, acc[a][c].w);
                            }
                    }
                }
            }
        }
    }
    __syncthreads();
    // ---- the slices' sums meet in shared memory, then the output (or the run's partial result) --------------------------------------------
    float* O = S;                                // [max(8, H)][dv]
    if (has_values) {
#pragma unroll
        for (int a = 0; a < kHW; ++a) {
            if (h0 + a >= H) continue;
#pragma unroll
            for (int c = 0; c < kC; ++c) {
                const int col = 4 * lane + 128 * c;
                float* dst = O + (slice * H + h0 + a) * dv + col;
                if (col < dv) *reinterpret_cast<float2*>(dst) = make_float2(acc[a][c].x, acc[a][c].y);
                if (col + 2 < dv) *reinterpret_cast<float2*>(dst + 2) = make_float2(acc[a][c].z, acc[a][c].w);
            }
        }
    }
    __syncthreads();
    const int half = dv >> 1;
    for (int e = threadIdx.x; e < H * half; e += 256) {
        const int h = e / half, m = e - h * half;
        float a = 0.f, b = 0.f;
        for (int s = 0; s < slices; ++s) { a += O[(s * H + h) * dv + m]; b += O[(s * H + h) * dv + m + half]; }
        if (A.splits > 1) {
            float* pp = A.part + (((int64_t)t * A.splits + split) * H + h) * (dv + 2);
            pp[m] = a; pp[m + half] = b;
            if (m == 0) { pp[dv] = ms[h]; pp[dv + 1] = ls[h]; }
            continue;
        }
        const float inv = 1.0f / ls[h];
        a *= inv; b *= inv;
        if (A.cos_t) {
            const float c = A.cos_t[(int64_t)pos * half + m], s = A.sin_t[(int64_t)pos * half + m];
            const float u = a * c + b * s;
            b = b * c - a * s; a = u;
        }
        TOut* op = static_cast<TOut*>(A.out) + ((int64_t)t * H + h) * dv;
        op[m] = from_f32<TOut>(a); op[m + half] = from_f32<TOut>(b);
    }
}

template <typename TOut>
__global__ void __launch_bounds__(64)
talking_merge_kernel(const float* __restrict__ part, const int32_t* __restrict__ positions, const float* __restrict__ cos_t, const float* __restrict__ sin_t,
                     TOut* __restrict__ out, int H, int dv, int splits) {
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x, h = blockIdx.y, half = dv >> 1;
    const float* p0 = part + ((int64_t)t * splits * H + h) * (dv + 2);
    const int64_t step = (int64_t)H * (dv + 2);
    float m = -INFINITY;
    for (int s = 0; s < splits; ++s) m = fmaxf(m, p0[s * step + dv]);
    float l = 0.f;
    for (int s = 0; s < splits; ++s) l += expf(p0[s * step + dv] - m) * p0[s * step + dv + 1];       // a run without keys has maximum -inf: weight 0
    const float inv = 1.0f / l;
    const int pos = positions[t];
    for (int i = threadIdx.x; i < half; i += 64) {
        float a = 0.f, b = 0.f;
        for (int s = 0; s < splits; ++s) {
            const float w = expf(p0[s * step + dv] - m);
            a = fmaf(w, p0[s * step + i], a); b = fmaf(w, p0[s * step + i + half], b);
        }
        a *= inv; b *= inv;
        if (cos_t) {
            const float c = cos_t[(int64_t)pos * half + i], s = sin_t[(int64_t)pos * half + i];
            const float u = a * c + b * s;
            b = b * c - a * s; a = u;
        }
        out[((int64_t)t * H + h) * dv + i] = from_f32<TOut>(a);
        out[((int64_t)t * H + h) * dv + i + half] = from_f32<TOut>(b);
    }
}

// ---- portions of prompts on tensor cores --------------------------------------------------------------------------------------------------------
struct TalkTcArgs {
    const __nv_bfloat16* q; const __nv_bfloat16* kc; const __nv_bfloat16* vc;
    const int32_t* block_tables; int table_width;
    const int32_t* cu_q; const int32_t* cu_k; int num_seqs;
    const float* talk; const float* cos_t; const float* sin_t;
    __nv_bfloat16* out;
    int H, G, dk, dv, bs;
    float scale_log2;
    int chunk, window, one_sink;
    int kst, vst;                                // key / value tiles kept in shared memory (1 or 2)
    int pk, pv;                                  // row pitches in bytes, multiples of 128
    int bs_shift;
};

constexpr int kTcRows = 8, kTcWarps = 16, kTcThreads = kTcWarps * 32;        // query rows and warps of a block

__device__ __forceinline__ void cp16(uint32_t dst, const void* src) { asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(dst), "l"(src) : "memory"); }
__device__ __forceinline__ void cp_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
__device__ __forceinline__ void cp_wait_all() { asm volatile("cp.async.wait_group 0;" ::: "memory"); }
__device__ __forceinline__ void mma_bf16(float (&d)[4], uint32_t a0, uint32_t a1, uint32_t a2, uint32_t a3, uint32_t b0, uint32_t b1) {
    // not volatile: a pure function of its operands, which the compiler may move between the loads that feed it
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a0), "r"(a1), "r"(a2), "r"(a3), "r"(b0), "r"(b1));
}
__device__ __forceinline__ void ldsm_x4_trans(uint32_t (&r)[4], uint32_t addr) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];" : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(addr));
}
__device__ __forceinline__ float exp2_fast(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) { const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi); return *reinterpret_cast<const uint32_t*>(&v); }

// kHW: heads per warp (16 warps), kKT: keys per tile, k128: keys and values of 128 entries (the addresses are then constants)
template <int kHW, int kKT, bool k128>
__global__ void __launch_bounds__(kTcThreads, 1)
talking_prefill_kernel(const TalkTcArgs A) {
    pdl_wait();
    pdl_trigger();
    constexpr int kMT = kKT / 16, kSP = kKT + 4;                       // 16-key pieces per tile; pitch of a score row
    constexpr int kHP = 16 * kHW, kSH = kTcRows * kSP + 4, kTP = kHP + 8;      // heads rounded up (rows of zeros); pitches of a head's scores and of the mixing matrix
    extern __shared__ __align__(1024) uint8_t smem_tc[];
    const int H = A.H, G = A.G, dk = k128 ? 128 : A.dk, dv = k128 ? 128 : A.dv, pk = k128 ? 256 : A.pk, pv = k128 ? 256 : A.pv, group = H / G;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    // which (sequence, 8-row tile) is this block?  the last tiles of a sequence see the most keys and start first
    int seq = -1, tile = 0, base = 0;
    for (int s = 0; s < A.num_seqs; ++s) {
        const int nt = (A.cu_q[s + 1] - A.cu_q[s] + kTcRows - 1) / kTcRows;
        if ((int)blockIdx.x < base + nt) { seq = s; tile = nt - 1 - ((int)blockIdx.x - base); break; }
        base += nt;
    }
    if (seq < 0) return;
    const int q_begin = A.cu_q[seq], qlen = A.cu_q[seq + 1] - q_begin, klen = A.cu_k[seq + 1] - A.cu_k[seq];
    const int q0 = tile * kTcRows, rows = min(kTcRows, qlen - q0), pos0 = klen - qlen + q0, last_pos = pos0 + rows - 1;
    const int key0 = first_visible(pos0, A.chunk, A.window);
    const int ntiles = (last_pos - key0) / kKT + 1;
    const int32_t* table = A.block_tables + (int64_t)seq * A.table_width;

    const int kbytes = G * kKT * pk, vbytes = G * kKT * pv;
    const uint32_t sbase = (uint32_t)__cvta_generic_to_shared(smem_tc);
    auto lds16 = [&](uint32_t a) { return *reinterpret_cast<const uint4*>(smem_tc + (a - sbase)); };
    const uint32_t sQ = sbase, sK = sQ + H * kTcRows * pk, sV = sK + A.kst * kbytes;
    float* S = reinterpret_cast<float*>(smem_tc + (sV - sbase) + A.vst * vbytes);                   // [2][kHP][kSH]: rows of kSP floats per query
    constexpr int sstage = kHP * kSH;
    __nv_bfloat16* tk = reinterpret_cast<__nv_bfloat16*>(S + 2 * sstage);                            // [kHP][kTP] the mixing matrix, zeros past H
    const int magic_k = (65536 + (dk >> 3) - 1) / (dk >> 3), magic_v = (65536 + (dv >> 3) - 1) / (dv >> 3);

    // a tile of keys (or values) of every kv head: a warp takes whole cache rows; rows past the last visible key repeat it (their weight is 0)
    auto load_tile = [&](const __nv_bfloat16* cache, int d, uint32_t dst, int pitch, int tl, bool values) {
        const int d8 = d >> 3, pieces = G * d8, magic = values ? magic_v : magic_k;                  // (p * magic) >> 16 = p / d8 exactly for p < 1024, d8 <= 32
        const __nv_bfloat16* rows_of[kKT / kTcWarps];
#pragma unroll
        for (int kk = 0; kk < kKT / kTcWarps; ++kk)
            rows_of[kk] = cache + (int64_t)cache_row(table, min(key0 + tl * kKT + warp + kTcWarps * kk, last_pos), A.bs, A.bs_shift) * (G * d);
#pragma unroll
        for (int kk = 0; kk < kKT / kTcWarps; ++kk) {
            const int key = warp + kTcWarps * kk;
            const __nv_bfloat16* src = rows_of[kk];
            if constexpr (k128) {                                      // a lane's pieces lie two kv heads apart, at the same place of their rows
                const int c = lane & 15, cs = values ? c ^ (key & 7) : c ^ ((key & 1) << 2);
                uint32_t at = dst + ((lane >> 4) * kKT + key) * 256 + cs * 16;
                src += lane * 8;
#pragma unroll 4
                for (int p = lane; p < pieces; p += 32, at += 2 * kKT * 256, src += 256) cp16(at, src);
                continue;
            }
            for (int p = lane; p < pieces; p += 32) {
                const int kv = (p * magic) >> 16, c = p - kv * d8;
                const int cs = values ? c ^ (key & 7) : c ^ ((key & 1) << 2);
                cp16(dst + (kv * kKT + key) * pitch + cs * 16, src + p * 8);
            }
        }
    };
    auto load_k = [&](int tl) { if (tl < ntiles) load_tile(A.kc, dk, sK + (A.kst == 2 ? (tl & 1) * kbytes : 0), pk, tl, false); };
    auto load_v = [&](int tl) { if (tl < ntiles) load_tile(A.vc, dv, sV + (A.vst == 2 ? (tl & 1) * vbytes : 0), pv, tl, true); };

    {
        const int d8 = dk >> 3;
        for (int r = warp; r < H * kTcRows; r += kTcWarps) {
            const int h = r >> 3, qr = r & 7;
            const __nv_bfloat16* src = A.q + ((int64_t)(q_begin + q0 + min(qr, rows - 1)) * H + h) * dk;
            for (int c = lane; c < d8; c += 32) cp16(sQ + r * pk + (c ^ ((qr & 1) << 2)) * 16, src + c * 8);
        }
    }
    load_k(0);
    load_v(0);
    if (A.kst == 2) load_k(1);
    cp_commit();
    if (A.talk)
        for (int i = threadIdx.x; i < kHP * kHP; i += kTcThreads) {
            const int h = i / kHP, x = i % kHP;
            tk[h * kTP + x] = __float2bfloat16_rn(h < H && x < H ? A.talk[h * H + x] : 0.f);
        }
    for (int i = threadIdx.x; i < (kHP - H) * kSH; i += kTcThreads) S[H * kSH + i] = S[sstage + H * kSH + i] = 0.f;

    const int h0 = warp * kHW;
    float o[kHW][8][4];
    float m[kHW], l[kHW];
    int kvh[kHW];                                                      // kv heads of this warp's heads
#pragma unroll
    for (int a = 0; a < kHW; ++a) {
        kvh[a] = min(h0 + a, H - 1) / group;
#pragma unroll
        for (int n = 0; n < 8; ++n) o[a][n][0] = o[a][n][1] = o[a][n][2] = o[a][n][3] = 0.f;
        m[a] = A.one_sink ? 0.f : -INFINITY;                           // the sink: a key of score 0 without a value, counted by one lane of the query's four
        l[a] = A.one_sink && t == 0 ? 1.f : 0.f;
    }

    // raw scores of this warp's heads for tile tl into score stage tl & 1.  The four lanes of a row take 16-byte pieces of it: both operands
    // permute the contraction index the same way, so no transposing load is needed.
    const uint32_t off_a = (uint32_t)((t ^ ((g & 1) << 2)) * 16), off_b = off_a ^ 64u;       // of the even and odd 32-entry parts of a row pair
    auto scores = [&](int tl) {
        if (h0 >= H) return;
        float acc[kHW][kMT][4] = {};
        const uint32_t kb = sK + (A.kst == 2 ? (tl & 1) * kbytes : 0);
#pragma unroll (k128 ? 4 : 1)
        for (int d = 0; d < (dk + 31) / 32; ++d) {
            const bool ok = k128 || (4 * d + t) * 8 < dk;
            const uint32_t off = ((d & 1) ? off_b : off_a) + (d >> 1) * 128;
            uint4 ka[kMT][2];
            int kv_loaded = -1;
#pragma unroll
            for (int a = 0; a < kHW; ++a) {
                const int h = min(h0 + a, H - 1), kv = kvh[a];         // a head past the last repeats it: nothing of it is stored
                if (a == 0 || kv != kv_loaded) {
                    kv_loaded = kv;
                    const uint32_t at = kb + (kv * kKT + g) * pk + off;
#pragma unroll
                    for (int mt = 0; mt < kMT; ++mt)
#pragma unroll
                        for (int e = 0; e < 2; ++e) ka[mt][e] = ok ? lds16(at + (mt * 16 + e * 8) * pk) : make_uint4(0u, 0u, 0u, 0u);
                }
                const uint4 qb = ok ? lds16(sQ + (h * kTcRows + g) * pk + off) : make_uint4(0u, 0u, 0u, 0u);
#pragma unroll
                for (int mt = 0; mt < kMT; ++mt) {
                    mma_bf16(acc[a][mt], ka[mt][0].x, ka[mt][1].x, ka[mt][0].y, ka[mt][1].y, qb.x, qb.y);
                    mma_bf16(acc[a][mt], ka[mt][0].z, ka[mt][1].z, ka[mt][0].w, ka[mt][1].w, qb.z, qb.w);
                }
            }
        }
        float* Sd = S + (tl & 1) * sstage;
#pragma unroll
        for (int a = 0; a < kHW; ++a) {
            if (h0 + a >= H) continue;
            float* r0 = Sd + (h0 + a) * kSH + 2 * t * kSP;
#pragma unroll
            for (int mt = 0; mt < kMT; ++mt) {
                r0[mt * 16 + g] = acc[a][mt][0];
                r0[kSP + mt * 16 + g] = acc[a][mt][1];
                r0[mt * 16 + g + 8] = acc[a][mt][2];
                r0[kSP + mt * 16 + g + 8] = acc[a][mt][3];
            }
        }
    };
    // score stage st: s'[h] = sum_g talk[h, g] s[g] for every (query, key) pair, in place, on the tensor cores without leaving 32 bits: the mixing matrix is exact in
    // 16 bits, a score is the sum of three 16-bit numbers (8 bits of its 24 each), their products are exact and are summed in f32.  A warp takes eight
    // neighbouring keys of one query at a time; nobody else touches those columns.
    auto mix = [&](int st) {
        if (!A.talk) return;
        constexpr int kTiles = kTcRows * kKT / 8;
#pragma unroll
        for (int nt = warp; nt < kTiles; nt += kTcWarps) {
            float* col = S + st * sstage + (nt / (kKT / 8)) * kSP + (nt % (kKT / 8)) * 8;
            float acc[kHW][4] = {};
#pragma unroll
            for (int ks = 0; ks < kHW; ++ks) {
                uint32_t part[3][2];
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    float x = col[(ks * 16 + 2 * t + 8 * e) * kSH + g], y = col[(ks * 16 + 2 * t + 8 * e + 1) * kSH + g];
#pragma unroll
                    for (int p = 0; p < 3; ++p) {
                        part[p][e] = pack_bf16(x, y);
                        x -= __uint_as_float(part[p][e] << 16);
                        y -= __uint_as_float(part[p][e] & 0xffff0000u);
                    }
                }
#pragma unroll
                for (int mt = 0; mt < kHW; ++mt) {
                    const uint32_t* w = reinterpret_cast<const uint32_t*>(tk + (mt * 16 + g) * kTP + ks * 16) + t;
                    const uint32_t a0 = w[0], a1 = w[4 * kTP], a2 = w[4], a3 = w[4 * kTP + 4];
#pragma unroll
                    for (int p = 2; p >= 0; --p) mma_bf16(acc[mt], a0, a1, a2, a3, part[p][0], part[p][1]);
                }
            }
            __syncwarp();
#pragma unroll
            for (int mt = 0; mt < kHW; ++mt) {
                float* r0 = col + (mt * 16 + g) * kSH + 2 * t;                 // rows past H stay zero: the matrix has rows of zeros there
                *reinterpret_cast<float2*>(r0) = make_float2(acc[mt][0], acc[mt][1]);
                *reinterpret_cast<float2*>(r0 + 8 * kSH) = make_float2(acc[mt][2], acc[mt][3]);
            }
        }
    };

    cp_wait_all();
    __syncthreads();
    scores(0);
    __syncthreads();                                                   // all warps are done with key tile 0
    if (A.kst == 2) load_k(2); else load_k(1);
    cp_commit();
    if (A.kst != 2) { cp_wait_all(); __syncthreads(); }
    uint32_t voff[4];                                                  // a lane's row and swizzled 16-byte piece of a value tile, for four neighbouring pairs of pieces
    {
        const int key = (lane & 7) + ((lane >> 4) << 3);
#pragma unroll
        for (int n = 0; n < 4; ++n) voff[n] = (uint32_t)(key * pv + (((n * 2 + ((lane >> 3) & 1)) ^ (key & 7)) << 4));
    }
    const int pos = pos0 + g, lo = first_visible(pos, A.chunk, A.window);       // of this lane's query in the second product
    const int lo_last = first_visible(last_pos, A.chunk, A.window);
    for (int i = 0; i < ntiles; ++i) {
        if (i + 1 < ntiles) scores(i + 1);
        mix(i & 1);
        cp_wait_all();
        __syncthreads();
        // keys two tiles on (three when two tiles are kept: the other one holds tile i + 2) and the next values travel while this tile is finished
        load_k(A.kst == 2 ? i + 3 : i + 2);
        if (A.vst == 2) load_v(i + 1);
        cp_commit();
        const float* Sd = S + (i & 1) * sstage;
        if (h0 < H) {
            uint32_t pb[kHW][kMT][2];
            const int jt = key0 + i * kKT;
            const bool whole = jt + kKT - 1 <= pos0 && jt >= lo_last;      // every key of the tile is seen by every row
#pragma unroll
            for (int a = 0; a < kHW; ++a) {
                const float* row = Sd + min(h0 + a, H - 1) * kSH + g * kSP;
                const int j0 = key0 + i * kKT + 2 * t;
                float v[kMT][4], mx = -INFINITY;
#pragma unroll
                for (int mt = 0; mt < kMT; ++mt) {
                    const float2 x = *reinterpret_cast<const float2*>(row + mt * 16 + 2 * t), y = *reinterpret_cast<const float2*>(row + mt * 16 + 2 * t + 8);
                    v[mt][0] = x.x; v[mt][1] = x.y; v[mt][2] = y.x; v[mt][3] = y.y;
                    v[mt][0] *= A.scale_log2; v[mt][1] *= A.scale_log2; v[mt][2] *= A.scale_log2; v[mt][3] *= A.scale_log2;
                }
                if (!whole) {
#pragma unroll
                    for (int mt = 0; mt < kMT; ++mt)
#pragma unroll
                        for (int e = 0; e < 4; ++e) {
                            const int j = j0 + mt * 16 + (e >> 1) * 8 + (e & 1);
                            if (j < lo || j > pos) v[mt][e] = -INFINITY;
                        }
                }
#pragma unroll
                for (int mt = 0; mt < kMT; ++mt) mx = fmaxf(mx, fmaxf(fmaxf(v[mt][0], v[mt][1]), fmaxf(v[mt][2], v[mt][3])));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                const float mn = fmaxf(m[a], mx), subtr = mn == -INFINITY ? 0.f : mn;
                const float corr = exp2_fast(m[a] - subtr);
                m[a] = mn;
                float sum = 0.f;
#pragma unroll
                for (int mt = 0; mt < kMT; ++mt) {
                    const float p0 = exp2_fast(v[mt][0] - subtr), p1 = exp2_fast(v[mt][1] - subtr), p2 = exp2_fast(v[mt][2] - subtr), p3 = exp2_fast(v[mt][3] - subtr);
                    sum += (p0 + p1) + (p2 + p3);
                    pb[a][mt][0] = pack_bf16(p0, p1); pb[a][mt][1] = pack_bf16(p2, p3);
                }
                l[a] = fmaf(l[a], corr, sum);
                if (__any_sync(0xffffffffu, corr != 1.f)) {                // some row's maximum has moved
                    const float c0 = __shfl_sync(0xffffffffu, corr, 8 * t), c1 = __shfl_sync(0xffffffffu, corr, 8 * t + 4);      // of the accumulators' queries 2t, 2t + 1
#pragma unroll
                    for (int n = 0; n < 8; ++n) { o[a][n][0] *= c0; o[a][n][1] *= c1; o[a][n][2] *= c0; o[a][n][3] *= c1; }
                }
            }
            const uint32_t vb = sV + (A.vst == 2 ? (i & 1) * vbytes : 0);
#pragma unroll
            for (int mt = 0; mt < kMT; ++mt) {
#pragma unroll
                for (int n = 0; n < 8; ++n) {
                    if (n * 16 >= dv) break;
                    const uint32_t off = voff[n & 3] + (n >> 2) * 128 + mt * 16 * pv;
                    uint32_t va[4];
                    int kv_loaded = -1;
#pragma unroll
                    for (int a = 0; a < kHW; ++a) {
                        const int kv = kvh[a];
                        if (a == 0 || kv != kv_loaded) { kv_loaded = kv; ldsm_x4_trans(va, vb + kv * kKT * pv + off); }
                        mma_bf16(o[a][n], va[0], va[1], va[2], va[3], pb[a][mt][0], pb[a][mt][1]);
                    }
                }
            }
        }
        if (A.kst != 2 || A.vst != 2) {                                // a single buffer: everybody is done with it, then it is filled again
            if (A.kst != 2) cp_wait_all();
            __syncthreads();
            if (A.vst != 2) { load_v(i + 1); cp_commit(); }
        }
    }
    cp_wait_all();
    __syncthreads();
    // ---- normalise, turn back, store: head by head through a warp's own rows of shared memory --------------------------------------------------
    const int op = ((dv + 31) & ~31) + 4;                              // floats; 8 query rows per warp
    float* os = reinterpret_cast<float*>(smem_tc) + warp * kTcRows * op;
    const int half = dv >> 1;
#pragma unroll
    for (int a = 0; a < kHW; ++a) {
        const int h = h0 + a;
        if (h >= H) continue;
        float lt = l[a];
        lt += __shfl_xor_sync(0xffffffffu, lt, 1);
        lt += __shfl_xor_sync(0xffffffffu, lt, 2);
        const float inv = lt > 0.f ? 1.0f / lt : 0.f;
        const float i0 = __shfl_sync(0xffffffffu, inv, 8 * t), i1 = __shfl_sync(0xffffffffu, inv, 8 * t + 4);
        __syncwarp();
#pragma unroll
        for (int n = 0; n < 8; ++n) {
            if (n * 16 >= dv) break;
            os[(2 * t) * op + n * 16 + g] = o[a][n][0] * i0; os[(2 * t + 1) * op + n * 16 + g] = o[a][n][1] * i1;
            os[(2 * t) * op + n * 16 + g + 8] = o[a][n][2] * i0; os[(2 * t + 1) * op + n * 16 + g + 8] = o[a][n][3] * i1;
        }
        __syncwarp();
        for (int r = 0; r < rows; ++r) {
            __nv_bfloat16* dst = A.out + ((int64_t)(q_begin + q0 + r) * H + h) * dv;
            for (int x = lane; x < half; x += 32) {
                float u = os[r * op + x], w = os[r * op + x + half];
                if (A.cos_t) {
                    const float c = A.cos_t[(int64_t)(pos0 + r) * half + x], sn = A.sin_t[(int64_t)(pos0 + r) * half + x];
                    const float u2 = u * c + w * sn;
                    w = w * c - u * sn; u = u2;
                }
                dst[x] = __float2bfloat16_rn(u); dst[x + half] = __float2bfloat16_rn(w);
            }
        }
    }
}

// the tile and stage choice of a shape: heads per warp, keys per tile, stages of keys and values, bytes of shared memory (0 = not taken)
struct TcPlan { int hw, kt, kst, vst, pk, pv; size_t smem; };
TcPlan tc_plan(int H, int G, int dk, int dv) {
    TcPlan none{0, 0, 0, 0, 0, 0, 0};
    if (H > 32 || H % G || dk % 8 || dv % 16 || dv > 128 || dk > 256 || (int64_t)G * (dk > dv ? dk : dv) / 8 > 1024) return none;
    const int hw = H <= 16 ? 1 : 2;
    const int pk = (dk * 2 + 127) / 128 * 128, pv = (dv * 2 + 127) / 128 * 128;
    const int tries[6][3] = {{32, 2, 2}, {32, 2, 1}, {16, 2, 2}, {16, 2, 1}, {32, 1, 1}, {16, 1, 1}};
    for (const auto& c : tries) {
        if (hw == 2 && c[0] != 16) continue;                          // the registers of two heads per warp hold one 16-key piece of scores
        size_t b = (size_t)H * kTcRows * pk + (size_t)c[1] * G * c[0] * pk + (size_t)c[2] * G * c[0] * pv + (size_t)2 * 16 * hw * (kTcRows * (c[0] + 4) + 4) * 4 +
                   (size_t)16 * hw * (16 * hw + 8) * 2;
        const size_t outb = (size_t)kTcWarps * kTcRows * ((dv + 31) / 32 * 32 + 4) * 4;
        if (b < outb) b = outb;
        if (b <= 227 * 1024) return TcPlan{hw, c[0], c[1], c[2], pk, pv, b};
    }
    return none;
}

// ---- few rows in 16 bits on tensor cores --------------------------------------------------------------------------------------------------------
// A row alone needs no exchange of scores: mixing commutes with the product, s'[h, j] = (sum_g talk[h, g] q[g]) . k_j summed kv head by kv head, so every head gets
// one mixed query as long as a whole cache row, q'[h] = (talk[h, g] q[g] summed over the heads g of each kv head), and the scores of all heads are one product of
// q' [H, G dk] with the cache rows.  A block per (row, run of keys), eight or sixteen warps, 64 keys per tile: a warp scores eight keys (cache rows read straight into the operand
// layout, four lanes per row in 16-byte pieces), a warp per head takes the online softmax, and a warp multiplies the weights of one kv head's heads with 64 value
// columns (eight neighbouring columns per lane from four rows, paired in registers; the column order of the product is a permutation undone at the store).
constexpr int kDecTile = 64, kDecSP = kDecTile + 4, kDecPP = kDecTile + 8;      // keys per tile, pitches of a score row (f32) and of a weight row (bf16)
constexpr int kDecHead = 4 * kDecTile * 8 + 96 * 4;                             // bytes ahead of the queries: a multiple of 128

// kMT: 16-head tiles; kW: warps, 8 or 16 (two warps then share eight keys' scores, half of the cache row each).  Every warp has one (kv head, 64 columns) unit of the values
template <int kMT, int kW>
__global__ void __launch_bounds__(kW * 32, 16 / kW)
talking_decode_kernel(const TalkArgs A) {
    pdl_wait();
    pdl_trigger();
    extern __shared__ __align__(128) uint8_t smem_dec[];
    const int H = A.H, G = A.G, dk = A.dk, dv = A.dv, group = H / G, row = G * dk, pq = (row * 2 + 127) / 128 * 128;
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t = lane & 3;
    int64_t* ph = reinterpret_cast<int64_t*>(smem_dec);                      // [4][64] cache rows of the keys of this tile and the ones ahead
    float* cs = reinterpret_cast<float*>(ph + 4 * kDecTile);                 // [32] correction of this tile, [32] maxima (base 2), [32] denominators
    float* ms = cs + 32; float* ls = ms + 32;
    uint8_t* qm = smem_dec + kDecHead;                                       // [16 kMT][pq] mixed queries, 16-byte pieces swizzled
    float* S = reinterpret_cast<float*>(qm + 16 * kMT * pq);                 // [kW / 8][16 kMT][kDecSP]
    __nv_bfloat16* P = reinterpret_cast<__nv_bfloat16*>(S + kW / 8 * 16 * kMT * kDecSP);       // [H + 16][kDecPP]
    const int tok = blockIdx.x, split = blockIdx.y;
    const int pos = A.positions[tok];
    const int lo = first_visible(pos, A.chunk, A.window);
    const int per = ((pos - lo + A.splits) / A.splits + kDecTile - 1) / kDecTile * kDecTile;
    const int jb = lo + split * per, je = min(pos + 1, jb + per);
    const int32_t* table = A.block_tables + (int64_t)A.token_seq[tok] * A.table_width;
    const __nv_bfloat16* kc = static_cast<const __nv_bfloat16*>(A.kc);
    const __nv_bfloat16* vc = static_cast<const __nv_bfloat16*>(A.vc);
    auto place = [&](int j0, int buf) {          // keys past the run's end stand for its first one (their weight is 0, what they read is finite)
        if (j0 < je && threadIdx.x < kDecTile) {
            const int j = j0 + threadIdx.x < je ? j0 + threadIdx.x : jb;
            ph[buf * kDecTile + threadIdx.x] = cache_row(table, j, A.bs, A.bs_shift);
        }
    };
    const float scale_log2 = A.scale * 1.4426950408889634f;
    const int all_blk = row / 32, kg = warp & 7;                             // this warp's group of eight keys and its 32-entry parts of their rows
    const int blk0 = kW == 16 ? (warp >> 3) * (all_blk - all_blk / 2) : 0, nblk = kW == 16 ? (warp >> 3 ? all_blk / 2 : all_blk - all_blk / 2) : all_blk;
    uint4 nx[4];                                 // the next pieces of this warp's eight keys travel while earlier ones are multiplied, across tiles too
    auto first_pieces = [&](int j0, int buf) {
        if (j0 + kg * 8 >= je || nblk == 0) return;
        const uint4* kr = reinterpret_cast<const uint4*>(kc + ph[buf * kDecTile + kg * 8 + g] * row) + t + blk0 * 4;
#pragma unroll
        for (int i = 0; i < 4; ++i) nx[i] = kr[min(i, nblk - 1) * 4];
    };
    if (jb < je) {
        place(jb, 0);
        place(jb + kDecTile, 1);
        __syncthreads();
        first_pieces(jb, 0);
        // mixed queries in 16-byte pieces, eight neighbouring entries of one head each
        const int pieces = row >> 3, parts = max(1, kW * 32 / pieces), per_part = (16 * kMT + parts - 1) / parts;
        auto put = [&](int h, int c, const float (&v)[8]) {
            *reinterpret_cast<uint4*>(qm + h * pq + ((c ^ ((h & 1) << 2)) << 4)) =
                make_uint4(pack_bf16(v[0], v[1]), pack_bf16(v[2], v[3]), pack_bf16(v[4], v[5]), pack_bf16(v[6], v[7]));
        };
        for (int i = threadIdx.x; i < pieces * parts; i += kW * 32) {
            const int c = i % pieces, part = i / pieces, kv = c * 8 / dk, d = c * 8 - kv * dk;
            const int ha = part * per_part, hb = min(16 * kMT, ha + per_part);
            const float* q0 = A.q + ((int64_t)tok * H + kv * group) * dk + d;
            if (group <= 4) {                    // the kv head's queries stay in registers for all the heads of this thread
                float qv[4][8];
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    const float4* q4 = reinterpret_cast<const float4*>(q0 + (int64_t)min(e, group - 1) * dk);
                    const float4 a = q4[0], b = q4[1];
                    qv[e][0] = a.x; qv[e][1] = a.y; qv[e][2] = a.z; qv[e][3] = a.w; qv[e][4] = b.x; qv[e][5] = b.y; qv[e][6] = b.z; qv[e][7] = b.w;
                }
#pragma unroll 4
                for (int h = ha; h < hb; ++h) {
                    float w[4], v[8] = {};
#pragma unroll
                    for (int e = 0; e < 4; ++e)
                        w[e] = e < group && h < H ? (A.talk ? A.talk[h * H + kv * group + e] : (kv * group + e == h ? 1.f : 0.f)) * scale_log2 : 0.f;
#pragma unroll
                    for (int e = 0; e < 4; ++e)
#pragma unroll
                        for (int x = 0; x < 8; ++x) v[x] = fmaf(w[e], qv[e][x], v[x]);
                    put(h, c, v);
                }
            } else {
                for (int h = ha; h < hb; ++h) {
                    float v[8] = {};
                    for (int e = 0; e < group && h < H; ++e) {
                        const float w = (A.talk ? A.talk[h * H + kv * group + e] : (kv * group + e == h ? 1.f : 0.f)) * scale_log2;
                        const float4* q4 = reinterpret_cast<const float4*>(q0 + (int64_t)e * dk);
                        const float4 a = q4[0], b = q4[1];
                        v[0] = fmaf(w, a.x, v[0]); v[1] = fmaf(w, a.y, v[1]); v[2] = fmaf(w, a.z, v[2]); v[3] = fmaf(w, a.w, v[3]);
                        v[4] = fmaf(w, b.x, v[4]); v[5] = fmaf(w, b.y, v[5]); v[6] = fmaf(w, b.z, v[6]); v[7] = fmaf(w, b.w, v[7]);
                    }
                    put(h, c, v);
                }
            }
        }
    }
    if (threadIdx.x < 32) {
        const bool sink = A.one_sink && split == 0;                          // a key of score 0 without a value, counted by the first run
        ms[threadIdx.x] = sink ? 0.f : -INFINITY;
        ls[threadIdx.x] = sink ? 1.f : 0.f;
    }
    const int cols = (dv + 63) / 64, units = G * cols;
    float o[8][4];
#pragma unroll
    for (int n = 0; n < 8; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    const int ukv = warp < units ? warp / cols : -1, ucol = (warp % cols) * 64 + g * 8;      // kv head and first column of this lane's eight
    __syncthreads();
    const uint8_t* qrow = qm + g * pq + (((uint32_t)t ^ ((g & 1) << 2)) << 4);       // piece t of an even 32-entry part; the odd parts' lie 64 bytes away
    const int odd = (g & 1) ? -64 : 64;
    for (int j0 = jb, it = 0; j0 < je; j0 += kDecTile, ++it) {
        const int64_t* pht = ph + (it & 3) * kDecTile;
        // ---- scores of eight keys ------------------------------------------------------------------------------------------------------------
        if (j0 + kg * 8 < je) {
            const uint4* kr = reinterpret_cast<const uint4*>(kc + pht[kg * 8 + g] * row) + t + blk0 * 4;
            float acc[kMT][4] = {};
            for (int b = 0; b < nblk; b += 4) {
                uint4 cur[4];
#pragma unroll
                for (int i = 0; i < 4; ++i) cur[i] = nx[i];
                if (b + 4 < nblk) {
#pragma unroll
                    for (int i = 0; i < 4; ++i) nx[i] = kr[min(b + 4 + i, nblk - 1) * 4];
                }
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    if (b + i >= nblk) break;
                    const uint8_t* qa = qrow + ((blk0 + b + i) >> 1) * 128 + (((blk0 + b + i) & 1) ? odd : 0);
#pragma unroll
                    for (int mt = 0; mt < kMT; ++mt) {
                        const uint4 x = *reinterpret_cast<const uint4*>(qa + mt * 16 * pq), y = *reinterpret_cast<const uint4*>(qa + (mt * 16 + 8) * pq);
                        mma_bf16(acc[mt], x.x, y.x, x.y, y.y, cur[i].x, cur[i].y);
                        mma_bf16(acc[mt], x.z, y.z, x.w, y.w, cur[i].z, cur[i].w);
                    }
                }
            }
#pragma unroll
            for (int mt = 0; mt < kMT; ++mt) {
                float* sd = S + ((warp >> 3) * 16 * kMT + mt * 16 + g) * kDecSP + kg * 8 + 2 * t;
                *reinterpret_cast<float2*>(sd) = make_float2(acc[mt][0], acc[mt][1]);
                *reinterpret_cast<float2*>(sd + 8 * kDecSP) = make_float2(acc[mt][2], acc[mt][3]);
            }
        }
        // the first half of the tile's values travels during the softmax: rows 2t, 2t + 1, 2t + 8, 2t + 9 of two sets of sixteen keys
        uint4 vr[2][4];
        auto fetch_v = [&](int ks, uint4 (&d)[4]) {
            const bool ok = ukv >= 0 && ucol < dv;
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int key = ks * 16 + 2 * t + (e & 1) + (e >> 1) * 8;
                d[e] = ok ? *reinterpret_cast<const uint4*>(vc + (pht[key] * G + ukv) * dv + ucol) : make_uint4(0u, 0u, 0u, 0u);
            }
        };
        fetch_v(0, vr[0]);
        fetch_v(1, vr[1]);
        first_pieces(j0 + kDecTile, (it + 1) & 3);
        __syncthreads();
        // ---- online softmax, a warp per head ----------------------------------------------------------------------------------------------------
        for (int h = warp; h < H; h += kW) {
            float a = S[h * kDecSP + lane], b = S[h * kDecSP + 32 + lane];
            if (kW == 16) { a += S[(16 * kMT + h) * kDecSP + lane]; b += S[(16 * kMT + h) * kDecSP + 32 + lane]; }
            if (j0 + lane >= je) a = -INFINITY;                              // (what a skipped group left there is not looked at)
            if (j0 + 32 + lane >= je) b = -INFINITY;
            const float m_old = ms[h], m_new = fmaxf(m_old, warp_max(fmaxf(a, b)));
            a = exp2f(a - m_new); b = exp2f(b - m_new);
            P[h * kDecPP + lane] = __float2bfloat16_rn(a);
            P[h * kDecPP + 32 + lane] = __float2bfloat16_rn(b);
            const float sum = warp_sum(a + b);
            __syncwarp();
            if (lane == 0) {
                const float corr = exp2f(m_old - m_new);
                cs[h] = corr; ms[h] = m_new;
                ls[h] = fmaf(ls[h], corr, sum);
            }
        }
        place(j0 + 2 * kDecTile, (it + 2) & 3);
        __syncthreads();
        // ---- values -----------------------------------------------------------------------------------------------------------------------------
        if (ukv >= 0) {
            const int hb = ukv * group;
            const float c0 = g < group ? cs[hb + g] : 0.f, c1 = g + 8 < group ? cs[hb + g + 8] : 0.f;
#pragma unroll
            for (int n = 0; n < 8; ++n) { o[n][0] *= c0; o[n][1] *= c0; o[n][2] *= c1; o[n][3] *= c1; }
#pragma unroll
            for (int ks = 0; ks < 4; ++ks) {
                if (j0 + ks * 16 >= je) break;
                const __nv_bfloat16* p0 = P + (hb + g) * kDecPP + ks * 16 + 2 * t;       // rows past the group belong to other heads: their products are not stored
                const __nv_bfloat16* p1 = p0 + 8 * kDecPP;
                const uint32_t a0 = *reinterpret_cast<const uint32_t*>(p0), a2 = *reinterpret_cast<const uint32_t*>(p0 + 8);
                const uint32_t a1 = *reinterpret_cast<const uint32_t*>(p1), a3 = *reinterpret_cast<const uint32_t*>(p1 + 8);
                uint4 r[4];
#pragma unroll
                for (int e = 0; e < 4; ++e) r[e] = vr[ks & 1][e];
                if (ks < 2) fetch_v(ks + 2, vr[ks & 1]);
                const uint32_t w[4][4] = {{r[0].x, r[0].y, r[0].z, r[0].w}, {r[1].x, r[1].y, r[1].z, r[1].w}, {r[2].x, r[2].y, r[2].z, r[2].w}, {r[3].x, r[3].y, r[3].z, r[3].w}};
#pragma unroll
                for (int n2 = 0; n2 < 4; ++n2) {         // columns 2 n2 and 2 n2 + 1 of the lane's eight: pair the rows' low halves, then their high halves
                    mma_bf16(o[2 * n2], a0, a1, a2, a3, __byte_perm(w[0][n2], w[1][n2], 0x5410), __byte_perm(w[2][n2], w[3][n2], 0x5410));
                    mma_bf16(o[2 * n2 + 1], a0, a1, a2, a3, __byte_perm(w[0][n2], w[1][n2], 0x7632), __byte_perm(w[2][n2], w[3][n2], 0x7632));
                }
            }
        }
    }
    __syncthreads();
    // ---- output or the run's partial result: accumulator n of a lane's queries' columns 2t, 2t + 1 is value column 8 (2t) + n, 8 (2t + 1) + n of its 64 -------------
    float* O = reinterpret_cast<float*>(qm);                                 // [H][dv]
    if (ukv >= 0) {
        const int base = ucol - g * 8;
#pragma unroll
        for (int n = 0; n < 8; ++n)
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int r = g + (e >> 1) * 8, col = base + 8 * (2 * t + (e & 1)) + n;
                if (r < group && col < dv) O[(ukv * group + r) * dv + col] = o[n][e];
            }
    }
    __syncthreads();
    const int half = dv >> 1;
    for (int e = threadIdx.x; e < H * half; e += kW * 32) {
        const int h = e / half, x = e - h * half;
        float a = O[h * dv + x], b = O[h * dv + x + half];
        if (A.splits > 1) {
            float* pp = A.part + (((int64_t)tok * A.splits + split) * H + h) * (dv + 2);
            pp[x] = a; pp[x + half] = b;
            if (x == 0) { pp[dv] = ms[h] * 0.6931471805599453f; pp[dv + 1] = ls[h]; }        // the merge takes natural exponents
            continue;
        }
        const float inv = 1.0f / ls[h];
        a *= inv; b *= inv;
        if (A.cos_t) {
            const float c = A.cos_t[(int64_t)pos * half + x], s = A.sin_t[(int64_t)pos * half + x];
            const float u = a * c + b * s;
            b = b * c - a * s; a = u;
        }
        __nv_bfloat16* op = static_cast<__nv_bfloat16*>(A.out) + ((int64_t)tok * H + h) * dv;
        op[x] = __float2bfloat16_rn(a); op[x + half] = __float2bfloat16_rn(b);
    }
}

// shared memory of the kernel above for these sizes, 0 when it does not take them
size_t decode_plan(int H, int G, int dk, int dv) {
    if (H > 32 || H % G || H / G > 16 || (G * dk) % 32 || dk % 8 || dv % 8 || G * ((dv + 63) / 64) > 16) return 0;
    const int mt = (H + 15) / 16, pq = (G * dk * 2 + 127) / 128 * 128;
    const int wide = G * ((dv + 63) / 64) > 8;                               // sixteen warps, one block per SM
    size_t b = (size_t)16 * mt * pq + (size_t)(1 + wide) * 16 * mt * kDecSP * 4 + (size_t)(H + 16) * kDecPP * 2;
    const size_t outb = (size_t)H * dv * 4;
    if (b < outb) b = outb;
    b += kDecHead;
    return b <= (wide ? 220 : 110) * 1024 ? b : 0;
}

int block_shift(int bs) {
    for (int i = 0; i < 20; ++i)
        if (bs == 1 << i) return i;
    return -1;
}

template <typename TC, typename TOut>
bool launch_rows(const TalkArgs& A, int T, size_t smem, cudaStream_t st) {
    const int hw = (A.H + 7) / 8;
    const dim3 grid(T, A.splits);
#define TR(HW, CC) do { ensure_dynamic_smem((const void*)talking_rows_kernel<TC, TOut, HW, CC>, (int)smem); \
        launch_pdl(talking_rows_kernel<TC, TOut, HW, CC>, grid, dim3(256), smem, st, A); return true; } while (0)
#define TRC(HW) do { if (A.dv <= 128) TR(HW, 1); if (A.dv <= 256) TR(HW, 2); return false; } while (0)
    if (hw == 1) TRC(1);
    if (hw == 2) TRC(2);
    if (hw <= 4) TRC(4);
    if (hw <= 8) TRC(8);
#undef TRC
#undef TR
    return false;
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

void talking_attention_rows(void* out, const float* q, const void* key_cache, const void* value_cache, const int32_t* block_tables, int32_t table_width,
                            const int32_t* token_seq, const int32_t* positions, const float* talk, const float* v_cos, const float* v_sin, int32_t num_tokens,
                            int32_t num_heads, int32_t num_kv_heads, int32_t dk, int32_t dv, int32_t block_size, float scale, int32_t chunk, int32_t window,
                            int32_t one_sink, int32_t splits, float* part, int32_t plain, int32_t cache_dtype, int32_t out_dtype, int64_t stream) {
    if (num_tokens == 0) return;
    B200_REQUIRE(out && q && key_cache && value_cache && block_tables && token_seq && positions && (v_cos == nullptr) == (v_sin == nullptr), kErrBadArg,
                 "talking_attention_rows: null pointer");
    B200_REQUIRE(num_heads > 0 && num_kv_heads > 0 && num_heads % num_kv_heads == 0 && dk > 0 && dv > 0 && dv % 2 == 0 && block_size > 0 && table_width > 0 &&
                 splits >= 1 && splits <= 65535 && (splits == 1 || part), kErrBadArg, "talking_attention_rows: bad sizes (an even value size; scratch for more than one run)");
    B200_REQUIRE(num_heads <= 64 && dv <= 256 && dk <= 1024, kErrUnsupported, "talking_attention_rows: %d heads > 64, value size %d > 256 or key size %d > 1024", num_heads, dv, dk);
    const size_t dec_smem = cache_dtype == B200_BF16 && out_dtype == B200_BF16 && plain == 0 && (((uintptr_t)q | (uintptr_t)key_cache | (uintptr_t)value_cache) & 15) == 0
                                ? decode_plan(num_heads, num_kv_heads, dk, dv) : 0;
    TalkArgs A{q, key_cache, value_cache, block_tables, table_width, token_seq, positions, talk, v_cos, v_sin, out, part, num_heads, num_kv_heads, dk, dv, block_size,
               scale, chunk, window, one_sink, splits, 32, 0, block_shift(block_size)};
    const int subs = num_kv_heads >= 8 ? 1 : num_kv_heads >= 4 ? 2 : 4;                 // 32-key pieces per tile: work for eight warps
    A.tile = 32 * subs;
    const int span = cache_dtype == B200_F32 ? 16 : 32;                                 // entries four lanes take at a time
    A.qpitch = (dk + span - 1) / span * span + 4;                                       // + 4: neighbouring heads' rows start on different banks
    const int pool = 2 * num_heads * A.tile > (num_heads < 8 ? 8 : num_heads) * dv ? 2 * num_heads * A.tile : (num_heads < 8 ? 8 : num_heads) * dv;
    const size_t floats = (size_t)num_heads * A.qpitch + ((pool + 3) & ~3) + ((3 * num_heads + 3) & ~3) + 4 * (size_t)A.tile + (size_t)num_heads * num_heads;
    const size_t smem = floats * sizeof(float);
    B200_REQUIRE(dec_smem > 0 || smem <= 227 * 1024, kErrUnsupported, "talking_attention_rows: %d heads of key size %d do not fit shared memory", num_heads, dk);
    cudaStream_t st = as_stream(stream);
    bool ok = false;
    if (dec_smem > 0) {
        const dim3 grid(num_tokens, splits);
        const int units = num_kv_heads * ((dv + 63) / 64);
#define TDK(MT, WW) do { ensure_dynamic_smem((const void*)talking_decode_kernel<MT, WW>, (int)dec_smem); \
        launch_pdl(talking_decode_kernel<MT, WW>, grid, dim3(WW * 32), dec_smem, st, A); } while (0)
        if (num_heads <= 16) { if (units <= 8) TDK(1, 8); else TDK(1, 16); }
        else { if (units <= 8) TDK(2, 8); else TDK(2, 16); }
#undef TDK
        ok = true;
    } else if (cache_dtype == B200_F32 && out_dtype == B200_F32) ok = launch_rows<float, float>(A, num_tokens, smem, st);
    else if (cache_dtype == B200_BF16 && out_dtype == B200_BF16) ok = launch_rows<__nv_bfloat16, __nv_bfloat16>(A, num_tokens, smem, st);
    else { set_error(kErrUnsupported, "talking_attention_rows: cache dtype %d / out dtype %d", cache_dtype, out_dtype); return; }
    B200_REQUIRE(ok, kErrUnsupported, "talking_attention_rows: no kernel for %d heads, value size %d", num_heads, dv);
    count_launch();
    if (splits > 1) {
        const dim3 grid(num_tokens, num_heads);
        if (out_dtype == B200_F32) launch_pdl(talking_merge_kernel<float>, grid, dim3(64), 0, st, (const float*)part, positions, v_cos, v_sin, (float*)out, num_heads, dv, splits);
        else launch_pdl(talking_merge_kernel<__nv_bfloat16>, grid, dim3(64), 0, st, (const float*)part, positions, v_cos, v_sin, (__nv_bfloat16*)out, num_heads, dv, splits);
        count_launch();
    }
    check_launch("talking_attention_rows");
}

int32_t talking_attention_prefill_supported(int32_t num_heads, int32_t num_kv_heads, int32_t dk, int32_t dv) {
    return num_heads > 0 && num_kv_heads > 0 && dk > 0 && dv > 0 && tc_plan(num_heads, num_kv_heads, dk, dv).smem > 0 ? 1 : 0;
}

void talking_attention_prefill(void* out, const void* q, const void* key_cache, const void* value_cache, const int32_t* block_tables, int32_t table_width,
                               const int32_t* cu_seqlens_q, const int32_t* cu_seqlens_k, const float* talk, const float* v_cos, const float* v_sin, int32_t num_seqs,
                               int32_t num_tokens, int32_t num_heads, int32_t num_kv_heads, int32_t dk, int32_t dv, int32_t block_size, float scale, int32_t chunk,
                               int32_t window, int32_t one_sink, int64_t stream) {
    if (num_tokens == 0 || num_seqs == 0) return;
    B200_REQUIRE(out && q && key_cache && value_cache && block_tables && cu_seqlens_q && cu_seqlens_k && (v_cos == nullptr) == (v_sin == nullptr), kErrBadArg,
                 "talking_attention_prefill: null pointer");
    B200_REQUIRE(num_heads > 0 && num_kv_heads > 0 && num_heads % num_kv_heads == 0 && dk > 0 && dv > 0 && block_size > 0 && table_width > 0, kErrBadArg,
                 "talking_attention_prefill: bad sizes");
    const TcPlan P = tc_plan(num_heads, num_kv_heads, dk, dv);
    B200_REQUIRE(P.smem > 0 && (((uintptr_t)q | (uintptr_t)key_cache | (uintptr_t)value_cache) & 15) == 0, kErrUnsupported,
                 "talking_attention_prefill: %d / %d heads of %d / %d (at most 32 heads, dk a multiple of 8, dv of 16 and <= 128)", num_heads, num_kv_heads, dk, dv);
    TalkTcArgs A{(const __nv_bfloat16*)q, (const __nv_bfloat16*)key_cache, (const __nv_bfloat16*)value_cache, block_tables, table_width, cu_seqlens_q, cu_seqlens_k,
                 num_seqs, talk, v_cos, v_sin, (__nv_bfloat16*)out, num_heads, num_kv_heads, dk, dv, block_size, scale * 1.4426950408889634f, chunk, window, one_sink,
                 P.kst, P.vst, P.pk, P.pv, block_shift(block_size)};
    cudaStream_t st = as_stream(stream);
    const dim3 grid((unsigned)(num_tokens / kTcRows + num_seqs));
#define TTC3(HW, KT, W) do { ensure_dynamic_smem((const void*)talking_prefill_kernel<HW, KT, W>, (int)P.smem); \
        launch_pdl(talking_prefill_kernel<HW, KT, W>, grid, dim3(kTcThreads), P.smem, st, A); } while (0)
#define TTC(HW, KT) do { if (dk == 128 && dv == 128) TTC3(HW, KT, true); else TTC3(HW, KT, false); } while (0)
    if (P.hw == 1) { if (P.kt == 32) TTC(1, 32); else TTC(1, 16); }
    else TTC(2, 16);
#undef TTC3
#undef TTC
    count_launch();
    check_launch("talking_attention_prefill");
}

}  // extern "C"
