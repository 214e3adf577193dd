// Grouped-query attention with mixed heads on tensor cores (bf16 mma.sync.m16n8k16, float softmax): head h applies
// sum_g T[h, g] * (head g's softmax weights) to the values of its own key/value head, so every head of a token runs in one CTA.  Scores are
// kept in units of log 2; the logarithmic distance penalty is r1 log2(1 + r2 distance) there.  Weights enter the value product as a two-term
// bf16 split (as in seq_attn_mma.cu).
//
//   * prompt form (talk_prompt_kernel): two CTAs take up to 256 rows (token, head) of one sequence and walk the keys twice.  The first walk
//     leaves every row's log-sum-exp (sink included) in registers; the second forms the normalised weights, mixes them across heads through
//     shared memory in float and multiplies them with the values.  The mixture needs normalised weights of all heads at once, which is why
//     one online pass does not do; with G key/value heads, the pass that keeps every head's weights apart (below) would cost G value products.
//   * decode form (talk_decode_kernel, every sequence brings one token): few rows and a long key range, so the keys are read ONCE: the
//     mixture being linear, every head's unmixed weights are applied to every key/value head's values, partial sums of the key splits go to a
//     workspace, and talk_merge_kernel normalises and mixes them.
#include "seq_attn_mma.cuh"
#include <math.h>
#include <algorithm>

namespace wf {
namespace seq {

namespace {

constexpr int TK_THREADS = 256, TK_WARPS = 8;
constexpr int TK_MAX_HEADS = 32, TK_UNITS = 16;      // heads; 16-row units of the prompt form (one per warp)

constexpr int TK_MAX_SPLITS = 32;

struct TalkParams {
    int ub, rp2, rp2_log, tq;    // prompt form: units per key/value head, rows per token (group size rounded up to a power of two), tokens per CTA
    int kt, nst;                 // decode form: keys per tile, staged tiles
    int ps_log;                  // log2 of the page size where that is a power of two, else -1
    int splits;
    float* part;                 // decode form: [n][splits] of { [H][G][dv] weighted values, [H] maximum, [H] sum }
};

__host__ __device__ inline size_t talk_part_floats(const GqaDims& D) { return (size_t)D.H * D.G * D.dv + 2 * D.H; }

// two-term bf16 split of a pair: hi = round(a, b), lo = round(rest)
__device__ __forceinline__ void split_pair(float a, float b, uint32_t& hi, uint32_t& lo) {
    const float ah = __bfloat162float(__float2bfloat16_rn(a)), bh = __bfloat162float(__float2bfloat16_rn(b));
    hi = pack_bf16(ah, bh);
    lo = pack_bf16(a - ah, b - bh);
}

// one tile of keys (or values) of every key/value head, rows padded with zeros to `dp` entries: dst [G][kt][dp + 8]
template <int THREADS>
__device__ __forceinline__ void stage_rows(const GqaDims& D, const PagedCache& pc, const int32_t* bt, int ps_log, uint32_t dst, size_t base, int d, int dp, int kt, int j0, int pos_last) {
    const int kc = dp / 8, rstep = THREADS / kc, part = threadIdx.x % kc, row0 = threadIdx.x / kc;
    if (row0 >= rstep) return;
    const bool col_ok = part * 8 < d;
    const int stride = dp + 8;
    for (int key = row0; key < kt; key += rstep) {
        const int j = j0 + key;
        const bool ok = j <= pos_last;
        const int jj = ok ? j : 0, pg = ps_log >= 0 ? jj >> ps_log : jj / pc.page_size, slot = jj - pg * pc.page_size;
        const __nv_bfloat16* src = (const __nv_bfloat16*)pc.pool + (size_t)bt[pg] * pc.page_stride + pc.layer_off + base + (size_t)slot * d + (col_ok ? part * 8 : 0);
        for (int g = 0; g < D.G; ++g) am_cp16(dst + (uint32_t)((g * kt + key) * stride + part * 8) * 2u, src + (size_t)g * pc.page_size * d, ok && col_ok);
    }
}

// ---- prompt form --------------------------------------------------------------------------------------------------------------------
// A cluster of two CTAs shares the rows of a tile and takes every other key tile each: partial maxima and sums are exchanged once between the
// walks, partial outputs once at the end (each CTA finishes half the rows), both through distributed shared memory.  That halves the longest
// chain of key tiles, which is what a causal prompt's running time hangs on.
constexpr int TP_THREADS = 512, TP_WARPS = 16, TP_CLUSTER = 2;

__device__ __forceinline__ void cluster_sync_all() {
    asm volatile("barrier.cluster.arrive.aligned;\n\tbarrier.cluster.wait.aligned;" ::: "memory");
}
__device__ __forceinline__ uint32_t cluster_rank() {
    uint32_t r;
    asm("mov.u32 %0, %%cluster_ctarank;" : "=r"(r));
    return r;
}
// two floats at shared-memory address `addr` of the cluster's CTA `rank`
__device__ __forceinline__ float2 peer_ld2(uint32_t addr, uint32_t rank) {
    uint32_t a;
    float2 v;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"(addr), "r"(rank));
    asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(a) : "memory");
    return v;
}

// shared memory, in order: keys, values [G][KT][XS] bf16; weights P float [rows][PS]; mixed weights bf16 [2][rows][WS]; mixture float
// [H][hp]; penalties float [2][H][pt]; row statistics float [rows][2].  The output exchange reuses it from the start.
template <int DKP, int DVP, int KT>
struct TalkPromptShared {
    static constexpr int KS = DKP + 8, VS = DVP + 8, XS = KS > VS ? KS : VS;      // row strides in elements
    static constexpr int PS = KT + 4, WS = KT + 8;                                 // weights: floats, bf16
    static size_t bytes(int G, int units, int H, int tq) {
        const size_t rows = (size_t)units * 16, b = (size_t)4 * G * KT * XS + rows * (PS * 4 + 2 * WS * 2) + ((size_t)H * ((H + 3) / 4 * 4) + (size_t)2 * H * (KT + tq) + 2 * rows) * 4;
        const size_t exchange = (size_t)(DVP / 8) * TP_THREADS * 8;
        return b > exchange ? b : exchange;
    }
};

template <int DKP, int DVP, int KT>
__global__ void __launch_bounds__(TP_THREADS, 1) __cluster_dims__(TP_CLUSTER, 1, 1)
    talk_prompt_kernel(Batch b, GqaDims D, const __nv_bfloat16* __restrict__ qn, PagedCache pc, __nv_bfloat16* __restrict__ out, TalkParams tp) {
    using SH = TalkPromptShared<DKP, DVP, KT>;
    constexpr int KS = SH::KS, VS = SH::VS, PS = SH::PS, WS = SH::WS, NKS = DKP / 16, NVT = DVP / 8, NST = KT / 8;
    extern __shared__ __align__(16) unsigned char smraw[];
    const int units = D.G * tp.ub, rows = units * 16, hp = (D.H + 3) / 4 * 4, pt = KT + tp.tq;
    __nv_bfloat16* buf0 = reinterpret_cast<__nv_bfloat16*>(smraw);                 // keys (first walk: even turns)
    __nv_bfloat16* buf1 = buf0 + (size_t)D.G * KT * SH::XS;                        // values (first walk: keys of odd turns)
    float* P = reinterpret_cast<float*>(buf1 + (size_t)D.G * KT * SH::XS);         // [rows][PS] normalised weights
    __nv_bfloat16* Wh = reinterpret_cast<__nv_bfloat16*>(P + (size_t)rows * PS);   // [rows][WS] mixed weights, high and low terms
    __nv_bfloat16* Wl = Wh + (size_t)rows * WS;
    float* Tt = reinterpret_cast<float*>(Wl + (size_t)rows * WS);                  // [H][hp]: Tt[g][h] = T[h, g]
    float* pen = Tt + D.H * hp;                                                    // [2][H][pt]
    float* stat = pen + 2 * D.H * pt;                                              // [rows][2]
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g4 = lane >> 2, t4 = lane & 3, rep = D.H / D.G;
    const uint32_t rank = cluster_rank();
    int sq = -1, tok0 = 0, ntok = 0;
    {
        int t = (int)((gridDim.x - 1 - blockIdx.x) / TP_CLUSTER);      // the last tiles of a sequence see the most keys: they start first
        for (int s = 0; s < b.nseq; ++s) {
            const int tiles = (b.seq_len[s] + tp.tq - 1) / tp.tq;
            if (t < tiles) { sq = s; tok0 = t * tp.tq; ntok = b.seq_len[s] - tok0 < tp.tq ? b.seq_len[s] - tok0 : tp.tq; break; }
            t -= tiles;
        }
    }
    if (sq < 0) return;                                    // both CTAs of the cluster
    const int flat0 = b.seq_start[sq] + tok0, pos0 = b.seq_pos0[sq] + tok0, pos_last = pos0 + ntok - 1;
    const int32_t* bt = pc.block_table + (size_t)b.seq_slot[sq] * pc.max_blocks;
    for (int e = tid; e < D.H * hp; e += TP_THREADS) { const int g = e / hp, h = e - g * hp; Tt[e] = h < D.H ? D.talk[h * D.H + g] : 0.f; }
    // the warp's unit: 16 rows of key/value head warp / ub; row r -> token r >> rp2_log, head of the group r & (rp2 - 1)
    const bool busy = warp < units;
    const int kv = busy ? warp / tp.ub : 0, base = (warp - kv * tp.ub) * 16;
    bool r_ok[2];
    int r_tk[2], r_head[2], r_lo[2];
    float r_lse[2];
    uint32_t qf[NKS][4];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        const int r = base + g4 + 8 * k, tk = r >> tp.rp2_log, hg = r & (tp.rp2 - 1);
        r_ok[k] = busy && tk < ntok && hg < rep;
        r_tk[k] = r_ok[k] ? tk : 0; r_head[k] = kv * rep + (r_ok[k] ? hg : 0);
        int lo = pos0 + r_tk[k] - D.window + 1;
        if (D.chunk > 0) { const int c0 = (pos0 + r_tk[k]) / D.chunk * D.chunk; if (c0 > lo) lo = c0; }
        r_lo[k] = lo;
        const __nv_bfloat16* q = qn + ((size_t)(flat0 + r_tk[k]) * D.H + r_head[k]) * D.d;
#pragma unroll
        for (int ks = 0; ks < NKS; ++ks)
#pragma unroll
            for (int hlf = 0; hlf < 2; ++hlf) {
                const int c = ks * 16 + hlf * 8 + 2 * t4;
                qf[ks][k + 2 * hlf] = r_ok[k] && c < D.d ? *reinterpret_cast<const uint32_t*>(q + c) : 0u;
            }
    }
    // tiles that every row of the warp sees whole need no mask
    const int wpos_min = pos0 + (busy ? base >> tp.rp2_log : 0);
    const int wtk_max = (base + 15) >> tp.rp2_log, wpos_max = pos0 + (wtk_max < ntok ? wtk_max : ntok - 1);
    int wlo_max = wpos_max - D.window + 1;
    if (D.chunk > 0) { const int c0 = wpos_max / D.chunk * D.chunk; if (c0 > wlo_max) wlo_max = c0; }
    const float scale2 = D.scale * LOG2E;
    int lo_all = pos0 - D.window + 1 > 0 ? pos0 - D.window + 1 : 0;
    if (D.chunk > 0) { const int c0 = pos0 / D.chunk * D.chunk; if (c0 > lo_all) lo_all = c0; }
    const int t_lo = lo_all / KT + (int)rank, t_hi = pos_last / KT;                // this CTA's tiles: t_lo, t_lo + 2, ...
    const uint32_t sb0 = smem_u32(buf0), sb1 = smem_u32(buf1);
    const size_t v_base = (size_t)D.G * pc.page_size * D.d;
    const int mi = lane >> 3, rr = lane & 7;
    // penalties of the tile whose first key is j0, by head and distance: entry e belongs to distance pos0 - j0 - (KT - 1) + e
    auto fill_pen = [&](float* dst, int j0) {
        if (!D.dist_r1) return;
        for (int e = tid; e < D.H * pt; e += TP_THREADS) {
            const int h = e / pt, dist = pos0 - j0 - (KT - 1) + (e - h * pt);
            dst[e] = D.dist_r1[h] * __log2f(fmaf(D.dist_r2[h], (float)max(dist, 0), 1.f));
        }
    };
    // scores of the warp's rows on the tile at kb whose first key is j0: penalised, masked, units of log 2
    auto unit_scores = [&](uint32_t kb, const float* pn, int j0, float (&s)[NST][4]) {
#pragma unroll
        for (int j = 0; j < NST; ++j) { s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f; }
        const uint32_t kbu = kb + (uint32_t)(kv * KT * KS) * 2u;
#pragma unroll
        for (int ks = 0; ks < NKS; ++ks)
#pragma unroll
            for (int jp = 0; jp < NST / 2; ++jp) {
                uint32_t kf[4];
                am_ldsm_x4(kf, kbu + (uint32_t)((jp * 16 + (mi >> 1) * 8 + rr) * KS + ks * 16 + (mi & 1) * 8) * 2u);
                am_mma(s[2 * jp], qf[ks], kf[0], kf[1]);
                am_mma(s[2 * jp + 1], qf[ks], kf[2], kf[3]);
            }
        const bool whole = j0 + KT - 1 <= wpos_min && j0 >= wlo_max;
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            const float* pr = pn + r_head[k] * pt + r_tk[k] + KT - 1 - 2 * t4;
            const int d0 = pos0 + r_tk[k] - j0 - 2 * t4, l0 = j0 + 2 * t4 - r_lo[k];
#pragma unroll
            for (int j = 0; j < NST; ++j)
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    const int kk = j * 8 + e;
                    const float v = fmaf(s[j][2 * k + e], scale2, D.dist_r1 ? -pr[-kk] : 0.f);
                    s[j][2 * k + e] = whole || (kk <= d0 && kk + l0 >= 0) ? v : -INFINITY;
                }
        }
    };
    // ---- first walk: log-sum-exp of every row
    {
        float m_run[2] = {-INFINITY, -INFINITY}, l_run[2] = {0.f, 0.f};
        fill_pen(pen, t_lo * KT);
        if (t_lo <= t_hi) stage_rows<TP_THREADS>(D, pc, bt, tp.ps_log, sb0, 0, D.d, DKP, KT, t_lo * KT, pos_last);
        am_commit();
        int odd = 0;
        for (int t = t_lo; t <= t_hi; t += TP_CLUSTER, odd ^= 1) {
            am_wait<0>();
            __syncthreads();
            if (t + TP_CLUSTER <= t_hi) {
                stage_rows<TP_THREADS>(D, pc, bt, tp.ps_log, odd ? sb0 : sb1, 0, D.d, DKP, KT, (t + TP_CLUSTER) * KT, pos_last);
                am_commit();
                fill_pen(pen + (odd ^ 1) * D.H * pt, (t + TP_CLUSTER) * KT);
            }
            if (!busy) continue;
            float s[NST][4];
            unit_scores(odd ? sb1 : sb0, pen + odd * D.H * pt, t * KT, s);
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                float mx = -INFINITY;
#pragma unroll
                for (int j = 0; j < NST; ++j) mx = fmaxf(mx, fmaxf(s[j][2 * k], s[j][2 * k + 1]));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
                mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
                const float mn = fmaxf(m_run[k], mx), ms = mn == -INFINITY ? 0.f : mn;
                float ls = 0.f;
#pragma unroll
                for (int j = 0; j < NST; ++j) ls += exp2f(s[j][2 * k] - ms) + exp2f(s[j][2 * k + 1] - ms);
                l_run[k] = l_run[k] * exp2f(m_run[k] - ms) + ls;          // nothing seen yet: exp2(-inf) = 0
                m_run[k] = mn;
            }
        }
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            l_run[k] += __shfl_xor_sync(0xffffffffu, l_run[k], 1);
            l_run[k] += __shfl_xor_sync(0xffffffffu, l_run[k], 2);
            if (busy && t4 == 0) *reinterpret_cast<float2*>(stat + 2 * (warp * 16 + g4 + 8 * k)) = make_float2(m_run[k], l_run[k]);
        }
        cluster_sync_all();                                // both CTAs' statistics are there; this CTA's buffers are free
#pragma unroll
        for (int k = 0; k < 2; ++k) {
            r_lse[k] = 0.f;
            if (!busy) continue;
            const float2 o = peer_ld2(smem_u32(stat + 2 * (warp * 16 + g4 + 8 * k)), rank ^ 1u);
            const float m = fmaxf(m_run[k], o.x), ms = m == -INFINITY ? 0.f : m;
            const float l = l_run[k] * exp2f(m_run[k] - ms) + o.y * exp2f(o.x - ms);
            // weights are exp2(score - lse): -log2 of what a weight 2^m would be multiplied by, the sink's share included
            if (r_ok[k]) r_lse[k] = m - log2f(am_inv_sum(D, r_head[k], m, l));
        }
        cluster_sync_all();                                // read: a CTA without tiles may go on to write its output exchange
    }
    // ---- second walk: weights, mixture, values
    float o[NVT][4];
#pragma unroll
    for (int j = 0; j < NVT; ++j) { o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f; }
    fill_pen(pen, t_lo * KT);
    if (t_lo <= t_hi) stage_rows<TP_THREADS>(D, pc, bt, tp.ps_log, sb0, 0, D.d, DKP, KT, t_lo * KT, pos_last);
    am_commit();
    const uint32_t wh = smem_u32(Wh), wl = smem_u32(Wl);
    constexpr int JQ = KT / 4;
    const int mix_items = hp / 4 * tp.tq * JQ;
    int odd = 0;
    for (int t = t_lo; t <= t_hi; t += TP_CLUSTER, odd ^= 1) {
        am_wait<0>();
        __syncthreads();                                   // the keys are there; everyone is done with the values and the mixed weights
        stage_rows<TP_THREADS>(D, pc, bt, tp.ps_log, sb1, v_base, D.dv, DVP, KT, t * KT, pos_last);
        am_commit();
        if (busy) {
            float s[NST][4];
            unit_scores(sb0, pen + odd * D.H * pt, t * KT, s);
#pragma unroll
            for (int j = 0; j < NST; ++j)
#pragma unroll
                for (int k = 0; k < 2; ++k)
                    *reinterpret_cast<float2*>(P + (size_t)(warp * 16 + g4 + 8 * k) * PS + j * 8 + 2 * t4) =
                        make_float2(exp2f(s[j][2 * k] - r_lse[k]), exp2f(s[j][2 * k + 1] - r_lse[k]));
        }
        __syncthreads();                                   // every head's weights are there; the keys are free
        if (t + TP_CLUSTER <= t_hi) {
            stage_rows<TP_THREADS>(D, pc, bt, tp.ps_log, sb0, 0, D.d, DKP, KT, (t + TP_CLUSTER) * KT, pos_last);
            fill_pen(pen + (odd ^ 1) * D.H * pt, (t + TP_CLUSTER) * KT);
        }
        am_commit();
        for (int it = tid; it < mix_items; it += TP_THREADS) {         // four heads of a token on four keys
            const int jq = it % JQ, tk = (it / JQ) % tp.tq, hb = it / (JQ * tp.tq);
            float a[4][4];
#pragma unroll
            for (int h = 0; h < 4; ++h) a[h][0] = a[h][1] = a[h][2] = a[h][3] = 0.f;
            const float* pr = P + (size_t)(tk << tp.rp2_log) * PS + jq * 4;
            const float* tr = Tt + hb * 4;
            for (int g = 0; g < D.G; ++g, pr += (size_t)tp.ub * 16 * PS) {
#pragma unroll 4
                for (int hg = 0; hg < rep; ++hg, tr += hp) {
                    const float4 p = *reinterpret_cast<const float4*>(pr + hg * PS), w = *reinterpret_cast<const float4*>(tr);
                    a[0][0] = fmaf(w.x, p.x, a[0][0]); a[0][1] = fmaf(w.x, p.y, a[0][1]); a[0][2] = fmaf(w.x, p.z, a[0][2]); a[0][3] = fmaf(w.x, p.w, a[0][3]);
                    a[1][0] = fmaf(w.y, p.x, a[1][0]); a[1][1] = fmaf(w.y, p.y, a[1][1]); a[1][2] = fmaf(w.y, p.z, a[1][2]); a[1][3] = fmaf(w.y, p.w, a[1][3]);
                    a[2][0] = fmaf(w.z, p.x, a[2][0]); a[2][1] = fmaf(w.z, p.y, a[2][1]); a[2][2] = fmaf(w.z, p.z, a[2][2]); a[2][3] = fmaf(w.z, p.w, a[2][3]);
                    a[3][0] = fmaf(w.w, p.x, a[3][0]); a[3][1] = fmaf(w.w, p.y, a[3][1]); a[3][2] = fmaf(w.w, p.z, a[3][2]); a[3][3] = fmaf(w.w, p.w, a[3][3]);
                }
            }
#pragma unroll
            for (int h4 = 0; h4 < 4; ++h4) {
                const int h = hb * 4 + h4;
                if (h >= D.H) break;
                uint2 hi, lo;
                split_pair(a[h4][0], a[h4][1], hi.x, lo.x);
                split_pair(a[h4][2], a[h4][3], hi.y, lo.y);
                const int g = h / rep;
                const size_t at = (size_t)(g * tp.ub * 16 + (tk << tp.rp2_log) + h - g * rep) * WS + jq * 4;
                *reinterpret_cast<uint2*>(Wh + at) = hi;
                *reinterpret_cast<uint2*>(Wl + at) = lo;
            }
        }
        am_wait<1>();
        __syncthreads();                                   // mixed weights and values are there
        if (busy) {
            const uint32_t vb = sb1 + (uint32_t)(kv * KT * VS) * 2u;
#pragma unroll
            for (int kk = 0; kk < KT / 16; ++kk) {
                uint32_t ph[4], pl[4];
                const uint32_t at = (uint32_t)((warp * 16 + (lane & 15)) * WS + kk * 16 + (lane >> 4) * 8) * 2u;
                am_ldsm_x4(ph, wh + at);
                am_ldsm_x4(pl, wl + at);
#pragma unroll
                for (int np = 0; np < NVT / 2; ++np) {
                    uint32_t vf[4];
                    am_ldsm_x4_trans(vf, vb + (uint32_t)((kk * 16 + (mi & 1) * 8 + rr) * VS + np * 16 + (mi >> 1) * 8) * 2u);
                    am_mma(o[2 * np], ph, vf[0], vf[1]);
                    am_mma(o[2 * np + 1], ph, vf[2], vf[3]);
                    am_mma(o[2 * np], pl, vf[0], vf[1]);
                    am_mma(o[2 * np + 1], pl, vf[2], vf[3]);
                }
            }
        }
    }
    am_wait<0>();
    // ---- each CTA of the cluster finishes half the rows (rank 0: rows g4, rank 1: rows g4 + 8) and hands the other half over
    __syncthreads();
    float* xch = reinterpret_cast<float*>(smraw);          // [NVT][threads][2]
#pragma unroll
    for (int j = 0; j < NVT; ++j)
        *reinterpret_cast<float2*>(xch + 2 * (j * TP_THREADS + tid)) = rank == 0 ? make_float2(o[j][2], o[j][3]) : make_float2(o[j][0], o[j][1]);
    cluster_sync_all();
    const bool ok = rank == 0 ? r_ok[0] : r_ok[1];
    if (ok) {
        __nv_bfloat16* dst = out + ((size_t)(flat0 + (rank == 0 ? r_tk[0] : r_tk[1])) * D.H + (rank == 0 ? r_head[0] : r_head[1])) * D.dv;
#pragma unroll
        for (int j = 0; j < NVT; ++j) {
            const int c = j * 8 + 2 * t4;
            if (c >= D.dv) continue;
            const float2 p = peer_ld2(smem_u32(xch + 2 * (j * TP_THREADS + tid)), rank ^ 1u);
            *reinterpret_cast<uint32_t*>(dst + c) = pack_bf16((rank == 0 ? o[j][0] : o[j][2]) + p.x, (rank == 0 ? o[j][1] : o[j][3]) + p.y);
        }
    }
    cluster_sync_all();                                    // the other CTA may still be reading this one's shared memory
}

// ---- decode form --------------------------------------------------------------------------------------------------------------------
// shared memory of the decode form, in order: keys [nst][G][kt][kp + 8], values [nst][G][kt][vp + 8], queries [G][rp][kp + 8] (all bf16; kp,
// vp: sizes rounded up to 16, rp: group size rounded up to 8), scores float [H][kt + 4], weights bf16 [2][16 MT][kt + 8], maximum, sum and
// correction float [3][H]
struct TalkDecodeShared {
    int kp, vp, rp, mt;
    size_t k_tile, v_tile, q, sc, w;
    __host__ __device__ TalkDecodeShared(const GqaDims& D, int kt) {
        kp = (D.d + 15) / 16 * 16; vp = (D.dv + 15) / 16 * 16; rp = (D.H / D.G + 7) / 8 * 8; mt = (D.H + 15) / 16;
        k_tile = (size_t)D.G * kt * (kp + 8) * 2; v_tile = (size_t)D.G * kt * (vp + 8) * 2; q = (size_t)D.G * rp * (kp + 8) * 2;
        sc = (size_t)D.H * (kt + 4) * 4; w = (size_t)mt * 16 * (kt + 8) * 2;
    }
    __host__ __device__ size_t bytes(const GqaDims& D, int nst) const { return nst * (k_tile + v_tile) + q + sc + 2 * w + (size_t)3 * D.H * 4; }
};

// MT: 16-row tiles of heads; IT: (key/value head, 16 value columns) items per warp
template <int MT, int IT>
__global__ void __launch_bounds__(TK_THREADS, MT * IT <= 10 ? 2 : 1) talk_decode_kernel(Batch b, GqaDims D, const __nv_bfloat16* __restrict__ qn, PagedCache pc, TalkParams tp) {
    extern __shared__ __align__(16) unsigned char smraw[];
    const TalkDecodeShared sh(D, tp.kt);
    const int KT = tp.kt, KS = sh.kp + 8, VS = sh.vp + 8, SS = KT + 4, WS = KT + 8, nks = sh.kp / 16, rep = D.H / D.G;
    unsigned char* ks_ = smraw;
    unsigned char* vs_ = ks_ + tp.nst * sh.k_tile;
    __nv_bfloat16* Q = reinterpret_cast<__nv_bfloat16*>(vs_ + tp.nst * sh.v_tile);
    float* Sc = reinterpret_cast<float*>(reinterpret_cast<unsigned char*>(Q) + sh.q);
    __nv_bfloat16* Wh = reinterpret_cast<__nv_bfloat16*>(reinterpret_cast<unsigned char*>(Sc) + sh.sc);
    __nv_bfloat16* Wl = reinterpret_cast<__nv_bfloat16*>(reinterpret_cast<unsigned char*>(Wh) + sh.w);
    float* hm = reinterpret_cast<float*>(reinterpret_cast<unsigned char*>(Wl) + sh.w);
    float *hl = hm + D.H, *hc = hl + D.H;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g4 = lane >> 2, t4 = lane & 3, mi = lane >> 3, rr = lane & 7;
    const int sq = blockIdx.x, split = blockIdx.y, tok = b.seq_start[sq], pos = b.seq_pos0[sq];
    const int32_t* bt = pc.block_table + (size_t)b.seq_slot[sq] * pc.max_blocks;
    int lo = pos - D.window + 1 > 0 ? pos - D.window + 1 : 0;
    if (D.chunk > 0) { const int c0 = pos / D.chunk * D.chunk; if (c0 > lo) lo = c0; }
    int t_lo = lo / KT, t_hi = pos / KT;
    {
        const int per = (t_hi - t_lo + tp.splits) / tp.splits;
        t_lo += split * per;
        if (t_lo + per - 1 < t_hi) t_hi = t_lo + per - 1;
    }
    const size_t v_base = (size_t)D.G * pc.page_size * D.d;
    const uint32_t sk = smem_u32(ks_), sv = smem_u32(vs_), sq_ = smem_u32(Q), wh = smem_u32(Wh), wl = smem_u32(Wl);
    auto stage = [&](int t, int bf) {
        stage_rows<TK_THREADS>(D, pc, bt, tp.ps_log, sk + (uint32_t)(bf * sh.k_tile), 0, D.d, sh.kp, KT, t * KT, pos);
        stage_rows<TK_THREADS>(D, pc, bt, tp.ps_log, sv + (uint32_t)(bf * sh.v_tile), v_base, D.dv, sh.vp, KT, t * KT, pos);
        am_commit();
    };
    if (tp.nst == 2 && t_lo <= t_hi) stage(t_lo, 0);
    for (int e = tid; e < D.G * sh.rp * sh.kp; e += TK_THREADS) {
        const int r = e / sh.kp, c = e - r * sh.kp, kv = r / sh.rp, hg = r - kv * sh.rp;
        Q[r * KS + c] = hg < rep && c < D.d ? qn[((size_t)tok * D.H + kv * rep + hg) * D.d + c] : __float2bfloat16_rn(0.f);
    }
    for (int e = tid; e < (MT * 16 - D.H) * WS; e += TK_THREADS) { Wh[D.H * WS + e] = __float2bfloat16_rn(0.f); Wl[D.H * WS + e] = __float2bfloat16_rn(0.f); }
    for (int h = tid; h < D.H; h += TK_THREADS) { hm[h] = -INFINITY; hl[h] = 0.f; }
    const float scale2 = D.scale * LOG2E;
    const int nc = sh.vp / 16, items = D.G * nc;
    float o[IT][MT][2][4];
#pragma unroll
    for (int i = 0; i < IT; ++i)
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int c = 0; c < 2; ++c) { o[i][m][c][0] = o[i][m][c][1] = o[i][m][c][2] = o[i][m][c][3] = 0.f; }
    for (int t = t_lo; t <= t_hi; ++t) {
        int bf = 0;
        if (tp.nst == 2) {
            bf = (t - t_lo) & 1;
            am_wait<0>();
            __syncthreads();                               // the tile is there; everyone is done with the other buffer
            if (t < t_hi) stage(t + 1, bf ^ 1);
        } else {
            __syncthreads();
            stage(t, 0);
            am_wait<0>();
            __syncthreads();
        }
        const uint32_t kb = sk + (uint32_t)(bf * sh.k_tile), vb = sv + (uint32_t)(bf * sh.v_tile);
        // ---- raw scores, keys as the M rows and the heads of one key/value head as 8-wide N tiles
        const int kgroups = KT / 16, nr = sh.rp / 8;
        for (int it = warp; it < D.G * kgroups * nr; it += TK_WARPS) {
            const int n8 = it % nr, kk = (it / nr) % kgroups, kv = it / (nr * kgroups);
            float s[2][4] = {{0.f, 0.f, 0.f, 0.f}, {0.f, 0.f, 0.f, 0.f}};
            const uint32_t ka = kb + (uint32_t)((kv * KT + kk * 16 + (mi & 1) * 8 + rr) * KS + (mi >> 1) * 8) * 2u;
            const uint32_t qa = sq_ + (uint32_t)((kv * sh.rp + n8 * 8 + rr) * KS + mi * 8) * 2u;
            int ks = 0;
            for (; ks + 1 < nks; ks += 2) {                // two k-steps per query load, two accumulation chains
                uint32_t kf[4], kg[4], qf[4];
                am_ldsm_x4(qf, qa + (uint32_t)ks * 32u);
                am_ldsm_x4(kf, ka + (uint32_t)ks * 32u);
                am_ldsm_x4(kg, ka + (uint32_t)ks * 32u + 32u);
                am_mma(s[0], kf, qf[0], qf[1]);
                am_mma(s[1], kg, qf[2], qf[3]);
            }
            if (ks < nks) {
                uint32_t kf[4], qf[4];
                am_ldsm_x4(qf, sq_ + (uint32_t)((kv * sh.rp + n8 * 8 + rr) * KS + ks * 16 + (mi & 1) * 8) * 2u);
                am_ldsm_x4(kf, ka + (uint32_t)ks * 32u);
                am_mma(s[0], kf, qf[0], qf[1]);
            }
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int hg = n8 * 8 + 2 * t4 + (e & 1), key = kk * 16 + g4 + 8 * (e >> 1);
                if (hg < rep) Sc[(kv * rep + hg) * SS + key] = s[0][e] + s[1][e];
            }
        }
        __syncthreads();
        // ---- online softmax, a lane per key, 32 / KT heads per warp at a time
        const int per = 32 / KT, lk = lane & (KT - 1);
        for (int h0 = warp * per; h0 < D.H; h0 += TK_WARPS * per) {
            const int h = h0 + lane / KT, hh = h < D.H ? h : D.H - 1;
            const int key = t * KT + lk, dist = pos - key;
            float v = -INFINITY;
            if (dist >= 0 && key >= lo) {
                const float pen = D.dist_r1 ? D.dist_r1[hh] * __log2f(fmaf(D.dist_r2[hh], (float)dist, 1.f)) : 0.f;
                v = fmaf(Sc[hh * SS + lk], scale2, -pen);
            }
            float mx = v;
            for (int x = KT / 2; x > 0; x >>= 1) mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, x));
            const float mo = hm[hh], mn = fmaxf(mo, mx), ms = mn == -INFINITY ? 0.f : mn;
            const float p = exp2f(v - ms);
            float ls = p;
            for (int x = KT / 2; x > 0; x >>= 1) ls += __shfl_xor_sync(0xffffffffu, ls, x);
            __syncwarp();
            if (h < D.H) {
                const __nv_bfloat16 ph = __float2bfloat16_rn(p);
                Wh[h * WS + lk] = ph;
                Wl[h * WS + lk] = __float2bfloat16_rn(p - __bfloat162float(ph));
                if (lk == 0) { const float c = exp2f(mo - ms); hc[h] = c; hl[h] = hl[h] * c + ls; hm[h] = mn; }
            }
        }
        __syncthreads();
        // ---- every head's weights on every key/value head's values
        float corr[MT][2];
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int k = 0; k < 2; ++k) { const int h = m * 16 + g4 + 8 * k; corr[m][k] = h < D.H ? hc[h] : 0.f; }
#pragma unroll
        for (int i = 0; i < IT; ++i)
#pragma unroll
            for (int m = 0; m < MT; ++m)
#pragma unroll
                for (int c = 0; c < 2; ++c) { o[i][m][c][0] *= corr[m][0]; o[i][m][c][1] *= corr[m][0]; o[i][m][c][2] *= corr[m][1]; o[i][m][c][3] *= corr[m][1]; }
        for (int kk = 0; kk < KT / 16; ++kk) {
            uint32_t ph[MT][4], pl[MT][4];
#pragma unroll
            for (int m = 0; m < MT; ++m) {
                const uint32_t at = (uint32_t)((m * 16 + (lane & 15)) * WS + kk * 16 + (lane >> 4) * 8) * 2u;
                am_ldsm_x4(ph[m], wh + at);
                am_ldsm_x4(pl[m], wl + at);
            }
#pragma unroll
            for (int i = 0; i < IT; ++i) {
                const int it = warp + i * TK_WARPS;
                if (it < items) {
                    const int kv = it / nc, cc = it - kv * nc;
                    uint32_t vf[4];
                    am_ldsm_x4_trans(vf, vb + (uint32_t)((kv * KT + kk * 16 + (mi & 1) * 8 + rr) * VS + cc * 16 + (mi >> 1) * 8) * 2u);
#pragma unroll
                    for (int m = 0; m < MT; ++m) {
                        am_mma(o[i][m][0], ph[m], vf[0], vf[1]);
                        am_mma(o[i][m][1], ph[m], vf[2], vf[3]);
                        am_mma(o[i][m][0], pl[m], vf[0], vf[1]);
                        am_mma(o[i][m][1], pl[m], vf[2], vf[3]);
                    }
                }
            }
        }
    }
    am_wait<0>();
    float* part = tp.part + ((size_t)sq * tp.splits + split) * talk_part_floats(D);
#pragma unroll
    for (int i = 0; i < IT; ++i) {
        const int it = warp + i * TK_WARPS;
        if (it >= items) continue;
        const int kv = it / nc, cc = it - kv * nc;
#pragma unroll
        for (int m = 0; m < MT; ++m)
#pragma unroll
            for (int k = 0; k < 2; ++k) {
                const int h = m * 16 + g4 + 8 * k;
                if (h >= D.H) continue;
#pragma unroll
                for (int c = 0; c < 2; ++c) {
                    const int col = cc * 16 + c * 8 + 2 * t4;
                    if (col < D.dv) *reinterpret_cast<float2*>(part + ((size_t)h * D.G + kv) * D.dv + col) = make_float2(o[i][m][c][2 * k], o[i][m][c][2 * k + 1]);
                }
            }
    }
    __syncthreads();
    float* ml = part + (size_t)D.H * D.G * D.dv;
    for (int h = tid; h < D.H; h += TK_THREADS) { ml[h] = hm[h]; ml[D.H + h] = hl[h]; }
}

// block per (token, key/value head, four of its query heads): normalise the source heads over the splits, mix, write; every partial result is
// read once.  blockDim = (values rounded up to 32, slices of the sum)
constexpr int TM_HEADS = 4;
__global__ void talk_merge_kernel(Batch b, GqaDims D, int splits, const float* __restrict__ parts, __nv_bfloat16* __restrict__ out) {
    extern __shared__ __align__(16) float cf[];            // [splits][H][TM_HEADS] factors, then [slices][TM_HEADS][dv] partial sums
    const int sq = blockIdx.x, kv = blockIdx.y, rep = D.H / D.G, h0 = kv * rep + blockIdx.z * TM_HEADS, tok = b.seq_start[sq];
    const int tid = threadIdx.y * blockDim.x + threadIdx.x, cnt = min(TM_HEADS, kv * rep + rep - h0);
    const size_t pf = talk_part_floats(D), mo = (size_t)D.H * D.G * D.dv;
    const float* p = parts + (size_t)sq * splits * pf;
    float* red = cf + splits * D.H * TM_HEADS;
    for (int g = tid; g < D.H; g += blockDim.x * blockDim.y) {
        float m = -INFINITY, l = 0.f;
        for (int s = 0; s < splits; ++s) m = fmaxf(m, p[s * pf + mo + g]);
        for (int s = 0; s < splits; ++s) l = fmaf(p[s * pf + mo + D.H + g], exp2f(p[s * pf + mo + g] - m), l);
        const float inv = am_inv_sum(D, g, m, l);
        float w[TM_HEADS];
#pragma unroll
        for (int k = 0; k < TM_HEADS; ++k) w[k] = k < cnt ? D.talk[(h0 + k) * D.H + g] * inv : 0.f;
        for (int s = 0; s < splits; ++s) {
            const float f = exp2f(p[s * pf + mo + g] - m);
            *reinterpret_cast<float4*>(cf + (s * D.H + g) * TM_HEADS) = make_float4(w[0] * f, w[1] * f, w[2] * f, w[3] * f);
        }
    }
    __syncthreads();
    const int c = threadIdx.x;
    float v[TM_HEADS] = {0.f, 0.f, 0.f, 0.f};
    if (c < D.dv) {
        const float* src = p + (size_t)kv * D.dv + c;
        const int total = splits * D.H;
#pragma unroll 4
        for (int e = threadIdx.y; e < total; e += blockDim.y) {
            const int s = e / D.H, g = e - s * D.H;
            const float x = src[s * pf + (size_t)g * D.G * D.dv];
            const float4 f = *reinterpret_cast<const float4*>(cf + e * TM_HEADS);
            v[0] = fmaf(f.x, x, v[0]); v[1] = fmaf(f.y, x, v[1]); v[2] = fmaf(f.z, x, v[2]); v[3] = fmaf(f.w, x, v[3]);
        }
#pragma unroll
        for (int k = 0; k < TM_HEADS; ++k) red[(threadIdx.y * TM_HEADS + k) * D.dv + c] = v[k];
    }
    __syncthreads();
    for (int e = tid; e < cnt * D.dv; e += blockDim.x * blockDim.y) {
        float r = 0.f;
        for (int y = 0; y < (int)blockDim.y; ++y) r += red[y * TM_HEADS * D.dv + e];
        out[((size_t)tok * D.H + h0) * D.dv + e] = __float2bfloat16_rn(r);
    }
}

constexpr size_t TK_SMEM = 227 * 1024 - 1024;

int rows_per_token(const GqaDims& D) { int r = 1; while (r < D.H / D.G) r <<= 1; return r; }
int prompt_units(const GqaDims& D) { return std::max(1, TK_UNITS / D.G); }     // per key/value head
int prompt_tokens(const GqaDims& D) { return prompt_units(D) * 16 / rows_per_token(D); }

template <int KT>
size_t prompt_bytes(const GqaDims& D) {
    const int u = D.G * prompt_units(D), tq = prompt_tokens(D);
    if (D.d <= 64) return D.dv <= 64 ? TalkPromptShared<64, 64, KT>::bytes(D.G, u, D.H, tq) : TalkPromptShared<64, 128, KT>::bytes(D.G, u, D.H, tq);
    return D.dv <= 64 ? TalkPromptShared<128, 64, KT>::bytes(D.G, u, D.H, tq) : TalkPromptShared<128, 128, KT>::bytes(D.G, u, D.H, tq);
}

// keys per tile of the prompt form (0: the sizes do not fit)
int prompt_keys(const GqaDims& D) {
    if (D.G * prompt_units(D) > TK_UNITS) return 0;
    return prompt_bytes<32>(D) <= TK_SMEM ? 32 : (prompt_bytes<16>(D) <= TK_SMEM ? 16 : 0);
}

template <int DKP, int DVP, int KT>
int prompt_launch(const Batch& b, const GqaDims& D, const void* qn, const PagedCache& pc, void* out, const TalkParams& tp, cudaStream_t s) {
    static DevOnce once;
    if (once.need() && cuda_check(cudaFuncSetAttribute(talk_prompt_kernel<DKP, DVP, KT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TK_SMEM), "attention shared memory")) return WF_ERR_CUDA;
    // every sequence's tokens are cut into tiles of tq; n / tq + nseq bounds their number (clusters beyond the last tile return at once)
    talk_prompt_kernel<DKP, DVP, KT><<<TP_CLUSTER * (b.n / tp.tq + b.nseq), TP_THREADS, prompt_bytes<KT>(D), s>>>(b, D, (const __nv_bfloat16*)qn, pc, (__nv_bfloat16*)out, tp);
    return launch_check(cudaGetLastError(), "talk_prompt");
}

template <int KT>
int prompt_dispatch(const Batch& b, const GqaDims& D, const void* qn, const PagedCache& pc, void* out, const TalkParams& tp, cudaStream_t s) {
    if (D.d <= 64) return D.dv <= 64 ? prompt_launch<64, 64, KT>(b, D, qn, pc, out, tp, s) : prompt_launch<64, 128, KT>(b, D, qn, pc, out, tp, s);
    return D.dv <= 64 ? prompt_launch<128, 64, KT>(b, D, qn, pc, out, tp, s) : prompt_launch<128, 128, KT>(b, D, qn, pc, out, tp, s);
}

// tile and ring depth of the decode form; false where the accumulators or the tiles do not fit
bool decode_shape(const GqaDims& D, int& kt, int& nst) {
    const int mt = (D.H + 15) / 16, items = D.G * ((D.dv + 15) / 16), it = (items + TK_WARPS - 1) / TK_WARPS;
    if (mt > 2 || it > (mt == 1 ? 16 : 8)) return false;
    // two blocks per SM hide each other's phases: the larger tile only where two of its blocks fit
    if (2 * (TalkDecodeShared(D, 32).bytes(D, 2) + 1024) <= 228 * 1024) { kt = 32; nst = 2; return true; }
    const int shapes[2][2] = {{16, 2}, {16, 1}};
    for (const auto& x : shapes)
        if (TalkDecodeShared(D, x[0]).bytes(D, x[1]) <= TK_SMEM) { kt = x[0]; nst = x[1]; return true; }
    return false;
}

template <int MT, int IT>
int decode_launch(const Batch& b, const GqaDims& D, const void* qn, const PagedCache& pc, const TalkParams& tp, cudaStream_t s) {
    static DevOnce once;
    if (once.need() && cuda_check(cudaFuncSetAttribute(talk_decode_kernel<MT, IT>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)TK_SMEM), "attention shared memory")) return WF_ERR_CUDA;
    talk_decode_kernel<MT, IT><<<dim3(b.nseq, tp.splits), TK_THREADS, TalkDecodeShared(D, tp.kt).bytes(D, tp.nst), s>>>(b, D, (const __nv_bfloat16*)qn, pc, tp);
    return launch_check(cudaGetLastError(), "talk_decode");
}

}  // namespace

bool talk_attn_mma_usable(const GqaDims& D, const PagedCache& pc) {
    const int rep = D.G > 0 ? D.H / D.G : 0;
    return D.talk && rep >= 1 && rep <= 16 && D.H <= TK_MAX_HEADS && D.G <= TK_UNITS && D.d % 8 == 0 && D.dv % 8 == 0 && D.d <= 128 && D.dv <= 128 && !D.v_is_k && D.softcap == 0.f && !D.rel &&
           D.dist_exp == 0.f && pc.layer_off % 8 == 0 && pc.page_stride % 8 == 0 && ((long long)pc.page_size * D.d) % 8 == 0 && prompt_keys(D) > 0;
}

size_t talk_attn_workspace(const GqaDims& D, int n, int splits) { return (size_t)n * splits * talk_part_floats(D) * sizeof(float); }

int launch_talk_attn_mma(const Batch& b, const GqaDims& D, const void* qn, const PagedCache& pc, void* out, float* workspace, int splits, cudaStream_t s) {
    if (b.n <= 0) return WF_OK;
    if (!talk_attn_mma_usable(D, pc)) { set_error("attention: the tensor-core form with mixed heads does not take these sizes"); return WF_ERR_UNSUPPORTED; }
    TalkParams tp{};
    tp.ps_log = -1;
    for (int k = 0; k < 30; ++k) if (pc.page_size == (1 << k)) tp.ps_log = k;
    if (b.n == b.nseq && workspace && decode_shape(D, tp.kt, tp.nst)) {
        tp.splits = std::max(1, std::min(splits, TK_MAX_SPLITS)); tp.part = workspace;
        const int mt = (D.H + 15) / 16, it = (D.G * ((D.dv + 15) / 16) + TK_WARPS - 1) / TK_WARPS;
        int rc;
        if (mt == 1) rc = it <= 2 ? decode_launch<1, 2>(b, D, qn, pc, tp, s) : it <= 4 ? decode_launch<1, 4>(b, D, qn, pc, tp, s) : it <= 8 ? decode_launch<1, 8>(b, D, qn, pc, tp, s)
                                                                                                                                             : decode_launch<1, 16>(b, D, qn, pc, tp, s);
        else rc = it <= 2 ? decode_launch<2, 2>(b, D, qn, pc, tp, s) : it <= 5 ? decode_launch<2, 5>(b, D, qn, pc, tp, s) : decode_launch<2, 8>(b, D, qn, pc, tp, s);
        if (rc) return rc;
        const int rep = D.H / D.G;
        const dim3 block((D.dv + 31) / 32 * 32, 8);
        talk_merge_kernel<<<dim3(b.nseq, D.G, (rep + TM_HEADS - 1) / TM_HEADS), block, ((size_t)tp.splits * D.H + (size_t)block.y * D.dv) * TM_HEADS * sizeof(float), s>>>(
            b, D, tp.splits, workspace, (__nv_bfloat16*)out);
        return launch_check(cudaGetLastError(), "talk_merge");
    }
    tp.ub = prompt_units(D); tp.rp2 = rows_per_token(D); tp.tq = prompt_tokens(D);
    while ((1 << tp.rp2_log) < tp.rp2) ++tp.rp2_log;
    return prompt_keys(D) == 32 ? prompt_dispatch<32>(b, D, qn, pc, out, tp, s) : prompt_dispatch<16>(b, D, qn, pc, out, tp, s);
}

}  // namespace seq
}  // namespace wf
