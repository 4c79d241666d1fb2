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
    int chunk, window, one_sink, splits, tile, qpitch;
};

__device__ __forceinline__ int first_visible(int pos, int chunk, int window) {
    int lo = chunk > 0 ? (pos / chunk) * chunk : 0;
    if (window > 0 && pos - window + 1 > lo) lo = pos - window + 1;
    return lo;
}

template <typename TC> struct Piece;             // a 16-byte piece of a cached row as floats
template <> struct Piece<float> {
    static constexpr int N = 4;
    static __device__ __forceinline__ void load(const float* p, float (&v)[4]) { const float4 r = *reinterpret_cast<const float4*>(p); v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w; }
};
template <> struct Piece<__nv_bfloat16> {
    static constexpr int N = 8;
    static __device__ __forceinline__ void load(const __nv_bfloat16* p, float (&v)[8]) {
        const uint4 r = *reinterpret_cast<const uint4*>(p);
        const uint32_t w[4] = {r.x, r.y, r.z, r.w};
#pragma unroll
        for (int i = 0; i < 4; ++i) { v[2 * i] = __uint_as_float(w[i] << 16); v[2 * i + 1] = __uint_as_float(w[i] & 0xffff0000u); }
    }
};
__device__ __forceinline__ float2 load_pair(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 load_pair(const __nv_bfloat16* p) {
    const uint32_t w = *reinterpret_cast<const uint32_t*>(p);
    return make_float2(__uint_as_float(w << 16), __uint_as_float(w & 0xffff0000u));
}

// kHW: heads a warp accumulates values for, kC: pairs of value columns per lane (columns 2 lane + 64 c and the next)
template <typename TC, typename TOut, int kHW, int kC>
__global__ void __launch_bounds__(256)
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
            ph[buf * KT + i] = (int64_t)table[j / A.bs] * A.bs + j % A.bs;
        }
    };
    if (jb < je) place(jb, 0);
    // value heads of this warp; with fewer than eight heads the warps share a head's keys
    const int slices = H < 8 ? 8 / H : 1;
    const int h0 = H < 8 ? warp % H : warp * kHW, slice = H < 8 ? warp / H : 0;
    const bool has_values = slice < slices && h0 < H;
    float2 acc[kHW][kC];
#pragma unroll
    for (int a = 0; a < kHW; ++a)
#pragma unroll
        for (int c = 0; c < kC; ++c) acc[a][c] = make_float2(0.f, 0.f);
    const bool whole = dk % N == 0;              // rows are whole 16-byte pieces
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
                for (int d0 = 0; d0 < dk; d0 += 4 * N) {
                    const int d = d0 + c4 * N;
                    float kv[4][N];
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        if (whole) {
                            if (d < dk) Piece<TC>::load(kp[i] + d, kv[i]);
                            else {
#pragma unroll
                                for (int e = 0; e < N; ++e) kv[i][e] = 0.f;
                            }
                        } else {
#pragma unroll
                            for (int e = 0; e < N; ++e) kv[i][e] = d + e < dk ? to_f32<TC>(kp[i][d + e]) : 0.f;
                        }
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
                for (int c = 0; c < kC; ++c) { acc[a][c].x *= corr; acc[a][c].y *= corr; }
            }
            for (int k4 = slice * 4; k4 < nsub * 32; k4 += slices * 4) {
                if (j0 + k4 >= je) break;
                float4 p4[kHW];
#pragma unroll
                for (int a = 0; a < kHW; ++a) p4[a] = h0 + a < H ? *reinterpret_cast<const float4*>(P + (h0 + a) * KT + k4) : make_float4(0.f, 0.f, 0.f, 0.f);
                int g_loaded = -1;
                float2 vv[4][kC];
#pragma unroll
                for (int a = 0; a < kHW; ++a) {
                    const int g = min(h0 + a, H - 1) / group;
                    if (g != g_loaded) {
                        g_loaded = g;
#pragma unroll
                        for (int i = 0; i < 4; ++i) {
                            const TC* vp = vc + (pht[k4 + i] * G + g) * dv;
#pragma unroll
                            for (int c = 0; c < kC; ++c) {
                                const int col = 2 * lane + 64 * c;
                                vv[i][c] = col < dv ? load_pair(vp + col) : make_float2(0.f, 0.f);
                            }
                        }
                    }
                    const float p[4] = {p4[a].x, p4[a].y, p4[a].z, p4[a].w};
#pragma unroll
                    for (int i = 0; i < 4; ++i)
#pragma unroll
                        for (int c = 0; c < kC; ++c) { acc[a][c].x = fmaf(p[i], vv[i][c].x, acc[a][c].x); acc[a][c].y = fmaf(p[i], vv[i][c].y, acc[a][c].y); }
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
                const int col = 2 * lane + 64 * c;
                if (col < dv) *reinterpret_cast<float2*>(O + (slice * H + h0 + a) * dv + col) = acc[a][c];
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

template <typename TC, typename TOut>
bool launch_rows(const TalkArgs& A, int T, size_t smem, cudaStream_t st) {
    const int hw = (A.H + 7) / 8, pairs = (A.dv + 63) / 64;
    const dim3 grid(T, A.splits);
#define TR(HW, CC) do { ensure_dynamic_smem((const void*)talking_rows_kernel<TC, TOut, HW, CC>, (int)smem); \
        launch_pdl(talking_rows_kernel<TC, TOut, HW, CC>, grid, dim3(256), smem, st, A); return true; } while (0)
#define TRC(HW) do { if (pairs == 1) TR(HW, 1); if (pairs == 2) TR(HW, 2); if (pairs <= 4) TR(HW, 4); return false; } while (0)
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
                            int32_t one_sink, int32_t splits, float* part, int32_t cache_dtype, int32_t out_dtype, int64_t stream) {
    if (num_tokens == 0) return;
    B200_REQUIRE(out && q && key_cache && value_cache && block_tables && token_seq && positions && (v_cos == nullptr) == (v_sin == nullptr), kErrBadArg,
                 "talking_attention_rows: null pointer");
    B200_REQUIRE(num_heads > 0 && num_kv_heads > 0 && num_heads % num_kv_heads == 0 && dk > 0 && dv > 0 && dv % 2 == 0 && block_size > 0 && table_width > 0 &&
                 splits >= 1 && splits <= 65535 && (splits == 1 || part), kErrBadArg, "talking_attention_rows: bad sizes (an even value size; scratch for more than one run)");
    B200_REQUIRE(num_heads <= 64 && dv <= 256 && dk <= 1024, kErrUnsupported, "talking_attention_rows: %d heads > 64, value size %d > 256 or key size %d > 1024", num_heads, dv, dk);
    TalkArgs A{q, key_cache, value_cache, block_tables, table_width, token_seq, positions, talk, v_cos, v_sin, out, part, num_heads, num_kv_heads, dk, dv, block_size,
               scale, chunk, window, one_sink, splits, 32, 0};
    const int subs = num_kv_heads >= 8 ? 1 : num_kv_heads >= 4 ? 2 : 4;                 // 32-key pieces per tile: work for eight warps
    A.tile = 32 * subs;
    const int span = cache_dtype == B200_F32 ? 16 : 32;                                 // entries four lanes take at a time
    A.qpitch = (dk + span - 1) / span * span + 4;                                       // + 4: neighbouring heads' rows start on different banks
    const int pool = 2 * num_heads * A.tile > (num_heads < 8 ? 8 : num_heads) * dv ? 2 * num_heads * A.tile : (num_heads < 8 ? 8 : num_heads) * dv;
    const size_t floats = (size_t)num_heads * A.qpitch + ((pool + 3) & ~3) + ((3 * num_heads + 3) & ~3) + 4 * (size_t)A.tile + (size_t)num_heads * num_heads;
    const size_t smem = floats * sizeof(float);
    B200_REQUIRE(smem <= 227 * 1024, kErrUnsupported, "talking_attention_rows: %d heads of key size %d do not fit shared memory", num_heads, dk);
    cudaStream_t st = as_stream(stream);
    bool ok = false;
    if (cache_dtype == B200_F32 && out_dtype == B200_F32) ok = launch_rows<float, float>(A, num_tokens, smem, st);
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

}  // extern "C"
