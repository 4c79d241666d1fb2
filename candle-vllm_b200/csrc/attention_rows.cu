// attention_rows.cu -- grouped-query softmax attention over the paged cache for rows taken one at a time (decoded tokens, short portions) on tensor cores, bf16:
// a sliding window with kept first tokens, capped scores, a softmax sink, one sigmoid gate per output entry.
//
// A row at position i sees the keys j <= i with i - j < window (window 0 = all) or j < keep_first; its visible positions are numbered 0 .. n - 1 (the kept ones
// that lie before the window, then the window), so the window's start costs nothing and no key outside is read.  A block owns one row, one key / value head with
// up to 16 of the query heads that share it (the 16 rows of the MMA tile) and one of `splits` runs of the visible keys; its eight warps take 16 keys at a time in
// turn, each with its own online softmax, and join at the end through shared memory.
//
// Keys and values are fetched in the operand layout of mma.m16n8k16, 16 bytes per lane and copy.  The contraction over the head does not care about the order of
// its terms, so the four lanes of a key row take 16 neighbouring bytes each (entries 32 c + 8 t ..) and the query fragments are put together in the same order.  A
// value fragment pairs two keys per register: a lane takes 16 bytes (columns 64 c + 8 g ..) of its four key rows and pairs them by byte permutes; the columns come out
// permuted, which the store undoes.  The copies are cp.async into a ring of three tiles whose places belong to one lane each: a lane reads back only what it
// asked for itself, so the ring needs no barrier and two tiles are always on their way.
#include <algorithm>

#include "common.cuh"

namespace b200 {
namespace {

constexpr int kRowWarps = 8, kRowThreads = kRowWarps * 32;
constexpr float kLog2e = 1.4426950408889634f;

__device__ __forceinline__ float ex2(float x) { float y; asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x)); return y; }
__device__ __forceinline__ void mma_bf16(float (&d)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3]) : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t pack_bf16(float lo, float hi) { __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi); return *reinterpret_cast<uint32_t*>(&v); }

constexpr int kRing = 3;
__device__ __forceinline__ void copy16(uint4* dst, const void* src, bool ok) {        // zeros where the source does not exist
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"((uint32_t)__cvta_generic_to_shared(dst)), "l"(src), "r"(ok ? 16 : 0) : "memory");
}

struct RowsArgs {
    void* out; int64_t ldo;
    const __nv_bfloat16* q; const __nv_bfloat16* kc; const __nv_bfloat16* vc;
    const int32_t* tables; int table_width;
    const int32_t* token_seq; const int32_t* positions;
    int T, H, G, dk, dv, block_size;
    float scale, softcap;
    int window, keep_first;
    const float* sink; const float* gate; int64_t ldg;
    int splits; float* part;            // splits > 1: [T, H, splits, dv + 2]: the unnormalised sum, then the maximum (in units of log2) and the weight sum
};

// the last step of one entry of a head's output: weight sum with the sink, gate, rounding
__device__ __forceinline__ void store_entry(const RowsArgs& A, int t, int h, int c, float v) {
    if (A.gate) v *= 1.0f / (1.0f + expf(-A.gate[(int64_t)t * A.ldg + (int64_t)h * A.dv + c]));
    static_cast<__nv_bfloat16*>(A.out)[(int64_t)t * A.ldo + (int64_t)h * A.dv + c] = __float2bfloat16_rn(v);
}

// kDK, kDV: key and value size rounded up to 64 or 128
template <int kDK, int kDV>
__global__ void __launch_bounds__(kRowThreads)
attention_rows_kernel(const RowsArgs A) {
    pdl_wait();
    pdl_trigger();
    constexpr int kKC = kDK / 32, kVC = kDV / 64;       // 16-byte loads per key row and lane; per value row and lane
    constexpr int kPieces = 2 * kKC + 4 * kVC;          // copies of a lane per tile
    extern __shared__ __align__(16) float sm[];         // the ring [warps][kRing][kPieces][32] of 16 bytes; then [warps][16][kDV] sums, maxima, weight sums
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31, g = lane >> 2, t4 = lane & 3;
    const int rep = A.H / A.G, head_groups = (rep + 15) / 16;
    const int t = blockIdx.x, kvh = blockIdx.y / head_groups, hg = blockIdx.y % head_groups, split = blockIdx.z;
    const int h0 = kvh * rep + hg * 16, heads = min(16, rep - hg * 16);
    const int pos = A.positions[t];
    const int32_t* table = A.tables + (int64_t)A.token_seq[t] * A.table_width;
    const int lo = A.window > 0 ? max(0, pos - A.window + 1) : 0;
    const int kept = min(A.keep_first, lo), visible = kept + pos - lo + 1;
    // runs of whole 16-key tiles
    const int tiles = (visible + 15) / 16, per = (tiles + A.splits - 1) / A.splits;
    const int tile0 = split * per, tile1 = min(tiles, tile0 + per);

    // query fragments, rows g and g + 8 = heads h0 + g, h0 + g + 8; register pair order follows the key loads: of the 32 entries of chunk c a lane holds 8 t4 .. + 7
    uint32_t qa[2 * kKC][4];
#pragma unroll
    for (int c = 0; c < kKC; ++c) {
        const int d = 32 * c + 8 * t4;
        const __nv_bfloat16* qr = A.q + ((int64_t)t * A.H + h0) * A.dk + d;
        const uint4 zero = make_uint4(0, 0, 0, 0);
        const uint4 lo4 = (g < heads && d < A.dk) ? *reinterpret_cast<const uint4*>(qr + (int64_t)g * A.dk) : zero;
        const uint4 hi4 = (g + 8 < heads && d < A.dk) ? *reinterpret_cast<const uint4*>(qr + (int64_t)(g + 8) * A.dk) : zero;
        qa[2 * c][0] = lo4.x; qa[2 * c][1] = hi4.x; qa[2 * c][2] = lo4.y; qa[2 * c][3] = hi4.y;
        qa[2 * c + 1][0] = lo4.z; qa[2 * c + 1][1] = hi4.z; qa[2 * c + 1][2] = lo4.w; qa[2 * c + 1][3] = hi4.w;
    }
    float o[kDV / 8][4];
#pragma unroll
    for (int i = 0; i < kDV / 8; ++i) o[i][0] = o[i][1] = o[i][2] = o[i][3] = 0.f;
    float m_lo = -INFINITY, m_hi = -INFINITY, l_lo = 0.f, l_hi = 0.f;
    const float scale_log2 = A.scale * kLog2e;
    const float cap_log2 = A.softcap * kLog2e, cap_in = A.softcap > 0.f ? 2.f * scale_log2 / A.softcap : 0.f;

    // where key n of the tile lives: one lane per key looks it up (keys past the end read the last one, their weight is zero)
    auto locate = [&](int tile) {
        const int n = min(tile * 16 + (lane & 15), visible - 1);
        const int j = n < kept ? n : lo + n - kept;
        return table[j / A.block_size] * A.block_size + j % A.block_size;
    };
    uint4* ring = reinterpret_cast<uint4*>(sm) + (int64_t)warp * kRing * kPieces * 32 + lane;
    auto fetch = [&](int tile, int stage) {
        if (tile < tile1) {
            const int slot = locate(tile);
            uint4* dst = ring + stage * kPieces * 32;
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int64_t s = __shfl_sync(0xffffffffu, slot, half * 8 + g);
                const __nv_bfloat16* kr = A.kc + (s * A.G + kvh) * A.dk;
#pragma unroll
                for (int c = 0; c < kKC; ++c) {
                    const int d = 32 * c + 8 * t4;
                    copy16(dst + (half * kKC + c) * 32, kr + (d < A.dk ? d : 0), d < A.dk);
                }
            }
#pragma unroll
            for (int r = 0; r < 4; ++r) {               // key rows 2 t4, 2 t4 + 1, 2 t4 + 8, 2 t4 + 9
                const int64_t s = __shfl_sync(0xffffffffu, slot, 2 * t4 + (r & 1) + (r >> 1) * 8);
                const __nv_bfloat16* vr = A.vc + (s * A.G + kvh) * A.dv;
#pragma unroll
                for (int c = 0; c < kVC; ++c) {
                    const int d = 64 * c + 8 * g;
                    copy16(dst + (2 * kKC + r * kVC + c) * 32, vr + (d < A.dv ? d : 0), d < A.dv);
                }
            }
        }
        asm volatile("cp.async.commit_group;" ::: "memory");           // an empty group past the last tile: the count of groups stays that of the tiles
    };
    int stage = 0;
#pragma unroll
    for (int i = 0; i < kRing - 1; ++i) fetch(tile0 + warp + i * kRowWarps, i);
    for (int tile = tile0 + warp; tile < tile1; tile += kRowWarps) {
        fetch(tile + (kRing - 1) * kRowWarps, stage == 0 ? kRing - 1 : stage - 1);         // the place read in the previous turn
        asm volatile("cp.async.wait_group %0;" ::"n"(kRing - 1) : "memory");
        const uint4* src = ring + stage * kPieces * 32;
        stage = stage == kRing - 1 ? 0 : stage + 1;
        float s[2][4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            s[half][0] = s[half][1] = s[half][2] = s[half][3] = 0.f;
#pragma unroll
            for (int c = 0; c < kKC; ++c) {
                const uint4 kb = src[(half * kKC + c) * 32];
                mma_bf16(s[half], qa[2 * c], kb.x, kb.y);
                mma_bf16(s[half], qa[2 * c + 1], kb.z, kb.w);
            }
        }
        float mx_lo = -INFINITY, mx_hi = -INFINITY;
#pragma unroll
        for (int half = 0; half < 2; ++half) {
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const bool in = tile * 16 + half * 8 + 2 * t4 + (e & 1) < visible;
                float v = s[half][e];
                // cap tanh(x) = cap - 2 cap / (1 + e^(2x)): the error is absolute, a few ulp of the cap
                v = cap_log2 > 0.f ? fmaf(-2.f * cap_log2, __fdividef(1.0f, 1.0f + ex2(fminf(v * cap_in, 120.f))), cap_log2) : v * scale_log2;
                s[half][e] = in ? v : -INFINITY;
                if (e < 2) mx_lo = fmaxf(mx_lo, s[half][e]);
                else mx_hi = fmaxf(mx_hi, s[half][e]);
            }
        }
        mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 1)); mx_lo = fmaxf(mx_lo, __shfl_xor_sync(0xffffffffu, mx_lo, 2));
        mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 1)); mx_hi = fmaxf(mx_hi, __shfl_xor_sync(0xffffffffu, mx_hi, 2));
        const float mn_lo = fmaxf(m_lo, mx_lo), mn_hi = fmaxf(m_hi, mx_hi);       // a tile of a run holds at least one visible key: finite
        const float c_lo = ex2(m_lo - mn_lo), c_hi = ex2(m_hi - mn_hi);
        m_lo = mn_lo; m_hi = mn_hi;
        l_lo *= c_lo; l_hi *= c_hi;
        uint32_t pa[4];
#pragma unroll
        for (int half = 0; half < 2; ++half) {
            const float p0 = ex2(s[half][0] - m_lo), p1 = ex2(s[half][1] - m_lo), p2 = ex2(s[half][2] - m_hi), p3 = ex2(s[half][3] - m_hi);
            l_lo += p0 + p1; l_hi += p2 + p3;
            pa[2 * half] = pack_bf16(p0, p1); pa[2 * half + 1] = pack_bf16(p2, p3);
        }
#pragma unroll
        for (int i = 0; i < kDV / 8; ++i) { o[i][0] *= c_lo; o[i][1] *= c_lo; o[i][2] *= c_hi; o[i][3] *= c_hi; }
#pragma unroll
        for (int c = 0; c < kVC; ++c) {
            const uint4 v0 = src[(2 * kKC + c) * 32], v1 = src[(2 * kKC + kVC + c) * 32], v2 = src[(2 * kKC + 2 * kVC + c) * 32], v3 = src[(2 * kKC + 3 * kVC + c) * 32];
            const uint32_t r0[4] = {v0.x, v0.y, v0.z, v0.w}, r1[4] = {v1.x, v1.y, v1.z, v1.w}, r2[4] = {v2.x, v2.y, v2.z, v2.w}, r3[4] = {v3.x, v3.y, v3.z, v3.w};
#pragma unroll
            for (int w = 0; w < 4; ++w) {               // columns 64 c + 8 g + 2 w and + 1
                mma_bf16(o[8 * c + 2 * w], pa, __byte_perm(r0[w], r1[w], 0x5410), __byte_perm(r2[w], r3[w], 0x5410));
                mma_bf16(o[8 * c + 2 * w + 1], pa, __byte_perm(r0[w], r1[w], 0x7632), __byte_perm(r2[w], r3[w], 0x7632));
            }
        }
    }
    l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 1); l_lo += __shfl_xor_sync(0xffffffffu, l_lo, 2);
    l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 1); l_hi += __shfl_xor_sync(0xffffffffu, l_hi, 2);

    // join the warps, over the ring once every warp is done with its tiles: accumulator i = 8 c + e, columns 2 t4 and 2 t4 + 1 of the fragment are entries 64 c + 16 t4 + e and 64 c + 16 t4 + 8 + e of the head
    __syncthreads();
    float* sums = sm;
    float* ms = sm + kRowWarps * 16 * kDV;
    float* ls = ms + kRowWarps * 16;
#pragma unroll
    for (int i = 0; i < kDV / 8; ++i) {
        const int d = 64 * (i >> 3) + 16 * t4 + (i & 7);
        float* r_lo = sums + (warp * 16 + g) * kDV;
        float* r_hi = r_lo + 8 * kDV;
        r_lo[d] = o[i][0]; r_lo[d + 8] = o[i][1];
        r_hi[d] = o[i][2]; r_hi[d + 8] = o[i][3];
    }
    if (t4 == 0) {
        ms[warp * 16 + g] = m_lo; ms[warp * 16 + g + 8] = m_hi;
        ls[warp * 16 + g] = l_lo; ls[warp * 16 + g + 8] = l_hi;
    }
    __syncthreads();
    for (int e = threadIdx.x; e < heads * kDV; e += kRowThreads) {
        const int r = e / kDV, c = e % kDV, h = h0 + r;
        if (c >= A.dv) continue;
        const bool whole = A.splits == 1;
        float m = whole && A.sink ? A.sink[h] * kLog2e : -INFINITY;
#pragma unroll
        for (int w = 0; w < kRowWarps; ++w) m = fmaxf(m, ms[w * 16 + r]);
        const float sub = m == -INFINITY ? 0.f : m;
        float l = whole && A.sink ? ex2(A.sink[h] * kLog2e - sub) : 0.f, v = 0.f;
#pragma unroll
        for (int w = 0; w < kRowWarps; ++w) {
            const float f = ex2(ms[w * 16 + r] - sub);
            l = fmaf(f, ls[w * 16 + r], l);
            v = fmaf(f, sums[(w * 16 + r) * kDV + c], v);
        }
        if (whole) {
            store_entry(A, t, h, c, v / l);
        } else {
            float* pr = A.part + (((int64_t)t * A.H + h) * A.splits + split) * (A.dv + 2);
            pr[c] = v;
            if (c == 0) { pr[A.dv] = m; pr[A.dv + 1] = l; }
        }
    }
}

// one block per (row, head): the runs of its keys joined, the sink added
__global__ void __launch_bounds__(128)
attention_rows_merge_kernel(const RowsArgs A) {
    pdl_wait();
    pdl_trigger();
    const int t = blockIdx.x, h = blockIdx.y;
    const float* pr = A.part + ((int64_t)t * A.H + h) * A.splits * (A.dv + 2);
    float m = A.sink ? A.sink[h] * kLog2e : -INFINITY;
    for (int s = 0; s < A.splits; ++s) m = fmaxf(m, pr[(int64_t)s * (A.dv + 2) + A.dv]);
    float l = A.sink ? ex2(A.sink[h] * kLog2e - m) : 0.f;
    for (int s = 0; s < A.splits; ++s) l = fmaf(ex2(pr[(int64_t)s * (A.dv + 2) + A.dv] - m), pr[(int64_t)s * (A.dv + 2) + A.dv + 1], l);
    for (int c = threadIdx.x; c < A.dv; c += 128) {
        float v = 0.f;
        for (int s = 0; s < A.splits; ++s) v = fmaf(ex2(pr[(int64_t)s * (A.dv + 2) + A.dv] - m), pr[(int64_t)s * (A.dv + 2) + c], v);
        store_entry(A, t, h, c, v / l);
    }
}

}  // namespace
}  // namespace b200

using namespace b200;

extern "C" {

int32_t paged_attention_rows_supported(int32_t num_heads, int32_t num_kv_heads, int32_t dk, int32_t dv) {
    return num_heads > 0 && num_kv_heads > 0 && num_heads % num_kv_heads == 0 && dk > 0 && dv > 0 && dk % 8 == 0 && dv % 8 == 0 && dk <= 128 && dv <= 128 &&
           num_kv_heads * ((num_heads / num_kv_heads + 15) / 16) <= 65535;
}

void paged_attention_rows(void* out, int64_t ld_out, const void* q, const void* key_cache, const void* value_cache, const int32_t* block_tables, int32_t table_width,
                          const int32_t* token_seq, const int32_t* positions, int32_t num_tokens, int32_t num_heads, int32_t num_kv_heads, int32_t dk, int32_t dv,
                          int32_t block_size, float scale, int32_t window, int32_t keep_first, float softcap, const float* sink, const float* gate, int64_t ld_gate,
                          int32_t splits, float* part, int64_t stream) {
    if (num_tokens == 0) return;
    B200_REQUIRE(out && q && key_cache && value_cache && block_tables && token_seq && positions, kErrBadArg, "paged_attention_rows: null pointer");
    B200_REQUIRE(paged_attention_rows_supported(num_heads, num_kv_heads, dk, dv), kErrUnsupported, "paged_attention_rows: %d / %d heads of %d and %d", num_heads, num_kv_heads, dk, dv);
    B200_REQUIRE(num_tokens > 0 && table_width > 0 && block_size > 0 && window >= 0 && keep_first >= 0 && softcap >= 0.f && ld_out >= (int64_t)num_heads * dv &&
                 (!gate || ld_gate >= (int64_t)num_heads * dv) && splits >= 1 && splits <= 65535 && (splits == 1 || part) && num_heads <= 65535, kErrBadArg,
                 "paged_attention_rows: bad sizes");
    B200_REQUIRE((((uintptr_t)q | (uintptr_t)key_cache | (uintptr_t)value_cache) & 15) == 0, kErrBadArg, "paged_attention_rows: q and caches start on 16-byte borders");
    const RowsArgs A{out, ld_out, (const __nv_bfloat16*)q, (const __nv_bfloat16*)key_cache, (const __nv_bfloat16*)value_cache, block_tables, table_width, token_seq, positions,
                     num_tokens, num_heads, num_kv_heads, dk, dv, block_size, scale, softcap, window, keep_first, sink, gate, ld_gate, splits, part};
    cudaStream_t st = as_stream(stream);
    const dim3 grid(num_tokens, num_kv_heads * ((num_heads / num_kv_heads + 15) / 16), splits);
#define PAR(DK, DV) do { \
        const int smem = std::max(kRowWarps * 16 * (DV + 2) * (int)sizeof(float), kRowWarps * kRing * (DK / 16 + DV / 16) * 512); \
        ensure_dynamic_smem(reinterpret_cast<const void*>(attention_rows_kernel<DK, DV>), smem); \
        launch_pdl(attention_rows_kernel<DK, DV>, grid, dim3(kRowThreads), (size_t)smem, st, A); } while (0)
    if (dk <= 64) { if (dv <= 64) PAR(64, 64); else PAR(64, 128); }
    else { if (dv <= 64) PAR(128, 64); else PAR(128, 128); }
#undef PAR
    count_launch();
    if (splits > 1) {
        launch_pdl(attention_rows_merge_kernel, dim3(num_tokens, num_heads), dim3(128), 0, st, A);
        count_launch();
    }
    check_launch("paged_attention_rows");
}

}  // extern "C"
