// Gated delta rule: a per-head matrix state S [d, dv] in float that every token first decays (one factor per head, or one per head and key
// row), then corrects along its key (u = beta (v - S^T k), S += k u^T) and finally reads with its query (o = S^T q).  The same kernel
// without the correction (u = beta v) is the state-space recurrence S = a S + dt B x^T, y = S^T C with k = B, q = C, v = x, beta = dt, and,
// with one decay per key row and beta = 1, gated linear attention S = diag(a) S + k v^T.
// The state is carried per sequence slot across steps.
#include "seq_attn_mma.cuh"      // ldmatrix / mma.sync wrappers

namespace wf {
namespace seq {

namespace {

// one block per token: unit-normalise the q and k heads in place, compute the write strength and the decay of every head
template <typename T>
__global__ void delta_prep_kernel(DeltaDims D, float* __restrict__ qkv, int ld, const float* __restrict__ a_raw, int lda, const float* __restrict__ b_raw,
                                  int ldb, const T* __restrict__ A_log, const T* __restrict__ dt_bias, float* __restrict__ beta, float* __restrict__ decay) {
    const int i = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    float* row = qkv + (size_t)i * ld;
    const float qscale = 1.f / sqrtf((float)D.d);
    for (int v = warp; v < 2 * D.Hk; v += nw) {          // vectors 0 .. Hk-1 are q heads, Hk .. 2Hk-1 are k heads
        float* x = row + (size_t)v * D.d;
        float ss = 0.f;
        for (int c = lane; c < D.d; c += 32) ss += x[c] * x[c];
        ss = warp_sum(ss);
        const float inv = (v < D.Hk ? qscale : 1.f) / sqrtf(ss + 1e-6f);
        for (int c = lane; c < D.d; c += 32) x[c] *= inv;
    }
    for (int h = threadIdx.x; h < D.H; h += blockDim.x) beta[(size_t)i * D.H + h] = sigmoid_f(b_raw[(size_t)i * ldb + h]);
    const int nd = D.vec_decay ? D.H * D.d : D.H;         // one decay per head, or per head and key channel
    for (int k = threadIdx.x; k < nd; k += blockDim.x) {
        const int h = D.vec_decay ? k / D.d : k;
        const float sp = softplus_f(a_raw[(size_t)i * lda + k] + to_f(dt_bias[k]));
        decay[(size_t)i * nd + k] = expf(-expf(to_f(A_log[h])) * sp);
    }
}

// state-space recurrence: the step size and the decay of every head
template <typename T>
__global__ void ssd_prep_kernel(int n, int H, const float* __restrict__ dt_raw, int ld, const T* __restrict__ A_log, const T* __restrict__ dt_bias,
                                float* __restrict__ step, float* __restrict__ decay) {
    const int k = blockIdx.x * blockDim.x + threadIdx.x;
    if (k >= n * H) return;
    const int i = k / H, h = k - i * H;
    const float z = dt_raw[(size_t)i * ld + h] + to_f(dt_bias[h]);
    const float sp = z > 20.f ? z : log1pf(expf(z));     // softplus without a clamp
    step[k] = sp;
    decay[k] = expf(-expf(to_f(A_log[h])) * sp);
}

// one block per (token, norm group): v = (o + D_h x) * silu(z), divided by the root mean square of the group, times the weight
template <typename T>
__global__ void ssd_post_kernel(int H, int dv, int groups, const float* __restrict__ o, const float* __restrict__ x, int ldx, const float* __restrict__ z, int ldz,
                                const T* __restrict__ Dskip, const T* __restrict__ w, float eps, T* __restrict__ y) {
    __shared__ float scratch[33];
    const int i = blockIdx.x, g = blockIdx.y;
    const int inner = H * dv, gw = inner / groups;
    float ss = 0.f;
    for (int c = g * gw + threadIdx.x; c < (g + 1) * gw; c += blockDim.x) {
        const float xv = x[(size_t)i * ldx + c];
        const float v = (o[(size_t)i * inner + c] + to_f(Dskip[c / dv]) * xv) * silu_f(z[(size_t)i * ldz + c]);
        ss = fmaf(v, v, ss);
    }
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)gw + eps);
    for (int c = g * gw + threadIdx.x; c < (g + 1) * gw; c += blockDim.x) {
        const float xv = x[(size_t)i * ldx + c];
        const float v = (o[(size_t)i * inner + c] + to_f(Dskip[c / dv]) * xv) * silu_f(z[(size_t)i * ldz + c]);
        y[(size_t)i * inner + c] = from_f<T>(v * inv * to_f(w[c]));
    }
}

constexpr int DR_THREADS = 128, DR_TT = 16;

__device__ __forceinline__ void cp_async16(void* smem_dst, const void* gsrc) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;" ::"r"(smem_u32(smem_dst)), "l"(gsrc) : "memory");
}

// chunked run of a linear recurrence: pass 0 = whole portions in order (no chunks); pass 1 = a block takes one chunk from a ZERO state and
// leaves its end state (and the product of its decays) in the workspace; pass 3 = a block takes one chunk from the start state that
// scan_prefix_kernel chained and writes the outputs.  Workspace entry of (sequence, chunk): seq_start / chunk + sequence + chunk, which
// never collides between sequences and stays below tokens / chunk + sequences.
struct ScanArgs { int pass = 0, chunk = 0, nchunks = 1; float* local = nullptr; float* start = nullptr; float* prod = nullptr;
                  int v4 = 0; };   // v4: every staged row starts 16-byte aligned and has a multiple of 4 entries (16-byte copies)

__device__ __forceinline__ void cp_async4(void* smem_dst, const void* gsrc) {
    asm volatile("cp.async.ca.shared.global [%0], [%1], 4;" ::"r"(smem_u32(smem_dst)), "l"(gsrc) : "memory");
}

// block = (sequence, head, 16 value columns); thread = (column, eighth of the key rows: DPT consecutive ones), its part of the column in registers.
// Tokens are taken 16 at a time: the next group's k / q / v / gates are copied into the other half of shared memory (cp.async)
// while the current group runs, so the per-token chain is only register math, 16-byte shared-memory reads and two quad reductions.
// DR_PARTS = 8 (16 columns per block): short per-token chains and twice the blocks, for portions of many tokens;
// DR_PARTS = 4 (32 columns): wider, better coalesced state rows, for single decoded tokens where the state traffic is the cost.
// VEC: the decay is a vector over the key rows (staged per token like k and q) instead of one number per token.
// DELTA: the write is corrected by what the state already holds along the key (the delta rule); without it u = beta v.
// NC: columns per thread (consecutive ones; 2 halves the shared-memory reads per multiply-add where there are columns and rows enough).
template <int DPT, int DR_PARTS, bool VEC, bool DELTA, int NC>
__global__ void __launch_bounds__(DR_THREADS) delta_rule_kernel(Batch b, DeltaDims D, const float* __restrict__ qkv, int ld,
                                                                         const float* __restrict__ beta, const float* __restrict__ decay,
                                                                         float* __restrict__ state, size_t slot_stride, float* __restrict__ o, ScanArgs sa) {
    constexpr int DR_COLS = DR_THREADS / DR_PARTS * NC;
    extern __shared__ __align__(16) float sm[];
    // A thread owns DPT consecutive key rows; a token's k / q / decay rows lie in shared memory with 4 floats of padding after every DPT, so
    // that the eight (or four) threads of a column read their parts as 16-byte vectors from distinct banks.
    constexpr int PS = DPT + 4, RS = DR_PARTS * PS;           // floats per part and per token row
    constexpr int tile_floats = (VEC ? 3 : 2) * DR_TT * RS + DR_TT * DR_COLS + 2 * DR_TT;   // k [TT][RS], q [TT][RS], v [TT][cols], beta [TT], decay [TT], vector decay [TT][RS]
    const int sq = sa.pass ? blockIdx.x / sa.nchunks : blockIdx.x, h = blockIdx.y, col0 = blockIdx.z * DR_COLS;
    const int tid = threadIdx.x, p = tid % DR_PARTS, jl = tid / DR_PARTS * NC, col = col0 + jl;
    const int dvs = D.dv + D.ones_col;                      // state and output columns: the values, and the all-ones column behind them
    const int kh = h / (D.H / D.Hk);
    int start = b.seq_start[sq], len = b.seq_len[sq];
    float* S = state + (size_t)b.seq_slot[sq] * slot_stride + (size_t)h * D.d * dvs;       // where the state is read ...
    float* S_out = S;                                                                        // ... and where it is left
    if (sa.pass) {
        const int c = blockIdx.x - sq * sa.nchunks;
        if (c * sa.chunk >= len) return;                                                     // the whole block: this sequence has fewer chunks
        const size_t entry = ((size_t)(start / sa.chunk + sq + c) * D.H + h) * D.d * dvs;
        S = sa.pass == 1 ? nullptr : sa.start + entry;
        S_out = sa.pass == 1 ? sa.local + entry : nullptr;
        if (!VEC && sa.pass == 1 && tid == 0 && blockIdx.z == 0) {                           // the chunk's decay product (one decay per head)
            float pr = 1.f;
            const int t1 = len - c * sa.chunk < sa.chunk ? len - c * sa.chunk : sa.chunk;
            for (int t = 0; t < t1; ++t) pr *= decay[(size_t)(start + c * sa.chunk + t) * D.H + h];
            sa.prod[(size_t)(start / sa.chunk + sq + c) * D.H + h] = pr;
        }
        start += c * sa.chunk;
        len = len - c * sa.chunk < sa.chunk ? len - c * sa.chunk : sa.chunk;
    }
    float s[NC][DPT];
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int m = 0; m < DPT; ++m) {
            const int i = p * DPT + m;
            s[c][m] = (S && col + c < dvs && i < D.d) ? S[(size_t)i * dvs + col + c] : 0.f;
        }
    const int q_off = (D.q_off >= 0 ? D.q_off : 0) + kh * D.d, k_off = (D.k_off >= 0 ? D.k_off : D.Hk * D.d) + kh * D.d,
              v_off = (D.v_off >= 0 ? D.v_off : 2 * D.Hk * D.d) + h * D.dv;
    auto stage = [&](int buf, int t0) {
        float* ks = sm + (size_t)buf * tile_floats;
        float* qs = ks + DR_TT * RS;
        float* vs = qs + DR_TT * RS;
        float* bs = vs + DR_TT * DR_COLS;
        float* gs = bs + DR_TT;
        float* gv = gs + DR_TT;
        const int tt = len - t0 < DR_TT ? len - t0 : DR_TT;
        if (sa.v4) {
            const int d4 = D.d >> 2;
            for (int idx = tid; idx < tt * d4; idx += blockDim.x) {
                const int t = idx / d4, c = (idx - t * d4) << 2;
                const int at = t * RS + c + (c / DPT) * 4;    // the padded place of rows c .. c + 3 (DPT is a multiple of 4: one part holds them)
                const float* row = qkv + (size_t)(start + t0 + t) * ld;
                cp_async16(ks + at, row + k_off + c);
                cp_async16(qs + at, row + q_off + c);
                if (VEC) cp_async16(gv + at, decay + ((size_t)(start + t0 + t) * D.H + h) * D.d + c);
            }
            for (int idx = tid; idx < tt * (DR_COLS / 4); idx += blockDim.x) {
                const int t = idx / (DR_COLS / 4), c = (idx % (DR_COLS / 4)) << 2;
                if (col0 + c < D.dv) cp_async16(vs + t * DR_COLS + c, qkv + (size_t)(start + t0 + t) * ld + v_off + col0 + c);
                else {
#pragma unroll
                    for (int k = 0; k < 4; ++k) vs[t * DR_COLS + c + k] = (D.ones_col && col0 + c + k == D.dv) ? 1.f : 0.f;
                }
            }
        } else {
            for (int idx = tid; idx < tt * D.d; idx += blockDim.x) {
                const int t = idx / D.d, c = idx - t * D.d;
                const int at = t * RS + c + (c / DPT) * 4;    // the padded place of row c
                const float* row = qkv + (size_t)(start + t0 + t) * ld;
                cp_async4(ks + at, row + k_off + c);
                cp_async4(qs + at, row + q_off + c);
                if (VEC) cp_async4(gv + at, decay + ((size_t)(start + t0 + t) * D.H + h) * D.d + c);
            }
            for (int idx = tid; idx < tt * DR_COLS; idx += blockDim.x) {
                const int t = idx / DR_COLS, c = idx % DR_COLS;
                if (col0 + c < D.dv) cp_async4(vs + idx, qkv + (size_t)(start + t0 + t) * ld + v_off + col0 + c);
                else vs[idx] = (D.ones_col && col0 + c == D.dv) ? 1.f : 0.f;
            }
        }
        if (tid < tt) {
            if (beta) cp_async4(bs + tid, beta + (size_t)(start + t0 + tid) * D.H + h); else bs[tid] = 1.f;
            if (!VEC) cp_async4(gs + tid, decay + (size_t)(start + t0 + tid) * D.H + h);
        }
        cp_async_commit();
    };
    if (len > 0) stage(0, 0);
    int buf = 0;
    for (int t0 = 0; t0 < len; t0 += DR_TT, buf ^= 1) {
        const int tt = len - t0 < DR_TT ? len - t0 : DR_TT;
        cp_async_wait<0>();
        __syncthreads();                                      // group t0 landed; everyone is done with the other half
        if (t0 + DR_TT < len) stage(buf ^ 1, t0 + DR_TT);
        const float* ks = sm + (size_t)buf * tile_floats;
        const float* qs = ks + DR_TT * RS;
        const float* vs = qs + DR_TT * RS;
        const float* bs = vs + DR_TT * DR_COLS;
        const float* gs = bs + DR_TT;
        const float* gv = gs + DR_TT;
        const int i0 = p * DPT;                               // this thread's first key row
        for (int t = 0; t < tt; ++t) {
            const float4* kt = reinterpret_cast<const float4*>(ks + t * RS + p * PS);
            const float4* qt = reinterpret_cast<const float4*>(qs + t * RS + p * PS);
            const float4* gt = reinterpret_cast<const float4*>(gv + t * RS + p * PS);
            const float g = VEC ? 1.f : gs[t];
            // rows at and beyond D.d hold a zero state and stay zero: what the padding or an unstaged row holds never reaches them
            if (VEC) {                                        // the rows decay first, each by its own factor
#pragma unroll
                for (int m4 = 0; m4 < DPT / 4; ++m4) {
                    const float4 gg = gt[m4];
                    const int i = i0 + 4 * m4;
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        if (i < D.d) s[c][4 * m4] *= gg.x;
                        if (i + 1 < D.d) s[c][4 * m4 + 1] *= gg.y;
                        if (i + 2 < D.d) s[c][4 * m4 + 2] *= gg.z;
                        if (i + 3 < D.d) s[c][4 * m4 + 3] *= gg.w;
                    }
                }
            }
            float u[NC];
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                float rs = 0.f;
                if (DELTA) {
                    float r[4] = {0.f, 0.f, 0.f, 0.f};        // four chains: the sum over this thread's rows is not one dependent sequence
#pragma unroll
                    for (int m4 = 0; m4 < DPT / 4; ++m4) {
                        const float4 kk = kt[m4];
                        const int i = i0 + 4 * m4;
                        if (i < D.d) r[0] = fmaf(s[c][4 * m4], kk.x, r[0]);
                        if (i + 1 < D.d) r[1] = fmaf(s[c][4 * m4 + 1], kk.y, r[1]);
                        if (i + 2 < D.d) r[2] = fmaf(s[c][4 * m4 + 2], kk.z, r[2]);
                        if (i + 3 < D.d) r[3] = fmaf(s[c][4 * m4 + 3], kk.w, r[3]);
                    }
                    rs = (r[0] + r[1]) + (r[2] + r[3]);
                    rs += __shfl_xor_sync(0xffffffffu, rs, 1);
                    rs += __shfl_xor_sync(0xffffffffu, rs, 2);
                    if (DR_PARTS == 8) rs += __shfl_xor_sync(0xffffffffu, rs, 4);
                }
                u[c] = bs[t] * (vs[t * DR_COLS + jl + c] - g * rs);
            }
            if (sa.pass == 1) {                               // only the end state is wanted: no read-out
#pragma unroll
                for (int m4 = 0; m4 < DPT / 4; ++m4) {
                    const float4 kk = kt[m4];
                    const int i = i0 + 4 * m4;
#pragma unroll
                    for (int c = 0; c < NC; ++c) {
                        if (i < D.d) s[c][4 * m4] = fmaf(kk.x, u[c], g * s[c][4 * m4]);
                        if (i + 1 < D.d) s[c][4 * m4 + 1] = fmaf(kk.y, u[c], g * s[c][4 * m4 + 1]);
                        if (i + 2 < D.d) s[c][4 * m4 + 2] = fmaf(kk.z, u[c], g * s[c][4 * m4 + 2]);
                        if (i + 3 < D.d) s[c][4 * m4 + 3] = fmaf(kk.w, u[c], g * s[c][4 * m4 + 3]);
                    }
                }
                continue;
            }
            float out[NC][4];
#pragma unroll
            for (int c = 0; c < NC; ++c) out[c][0] = out[c][1] = out[c][2] = out[c][3] = 0.f;
#pragma unroll
            for (int m4 = 0; m4 < DPT / 4; ++m4) {
                const float4 kk = kt[m4], qq = qt[m4];
                const int i = i0 + 4 * m4;
#pragma unroll
                for (int c = 0; c < NC; ++c) {
                    if (i < D.d) { s[c][4 * m4] = fmaf(kk.x, u[c], g * s[c][4 * m4]); out[c][0] = fmaf(s[c][4 * m4], qq.x, out[c][0]); }
                    if (i + 1 < D.d) { s[c][4 * m4 + 1] = fmaf(kk.y, u[c], g * s[c][4 * m4 + 1]); out[c][1] = fmaf(s[c][4 * m4 + 1], qq.y, out[c][1]); }
                    if (i + 2 < D.d) { s[c][4 * m4 + 2] = fmaf(kk.z, u[c], g * s[c][4 * m4 + 2]); out[c][2] = fmaf(s[c][4 * m4 + 2], qq.z, out[c][2]); }
                    if (i + 3 < D.d) { s[c][4 * m4 + 3] = fmaf(kk.w, u[c], g * s[c][4 * m4 + 3]); out[c][3] = fmaf(s[c][4 * m4 + 3], qq.w, out[c][3]); }
                }
            }
#pragma unroll
            for (int c = 0; c < NC; ++c) {
                float os = (out[c][0] + out[c][1]) + (out[c][2] + out[c][3]);
                os += __shfl_xor_sync(0xffffffffu, os, 1);
                os += __shfl_xor_sync(0xffffffffu, os, 2);
                if (DR_PARTS == 8) os += __shfl_xor_sync(0xffffffffu, os, 4);
                if (p == 0 && col + c < dvs) o[((size_t)(start + t0 + t) * D.H + h) * dvs + col + c] = os * D.o_scale;
            }
        }
    }
    if (!S_out) return;
#pragma unroll
    for (int c = 0; c < NC; ++c)
#pragma unroll
        for (int m = 0; m < DPT; ++m) {
            const int i = p * DPT + m;
            if (col + c < dvs && i < D.d) S_out[(size_t)i * dvs + col + c] = s[c][m];
        }
}

// thread per (sequence, head, state element): chains the chunks' start states from the slot's state and leaves the end state in the slot.
// prod has one entry per (chunk, head), or (d > 0) one per (chunk, head, key row) of dd / d state columns each
__global__ void scan_prefix_kernel(Batch b, int H, int dd, int chunk, float* __restrict__ state, size_t slot_stride, const float* __restrict__ local,
                                   float* __restrict__ startws, const float* __restrict__ prod, int d) {
    const int sq = blockIdx.x, h = blockIdx.y, e = blockIdx.z * blockDim.x + threadIdx.x;
    if (e >= dd) return;
    const int len = b.seq_len[sq], nc = (len + chunk - 1) / chunk, base = b.seq_start[sq] / chunk + sq;
    float* Sp = state + (size_t)b.seq_slot[sq] * slot_stride + (size_t)h * dd + e;
    float S = *Sp;
    for (int c = 0; c < nc; ++c) {
        const size_t entry = (size_t)(base + c) * H + h;
        startws[entry * dd + e] = S;
        S = fmaf(d > 0 ? prod[entry * d + e / (dd / d)] : prod[entry], S, local[entry * dd + e]);
    }
    *Sp = S;
}

// thread per (sequence and chunk, head and key row): the product of the chunk's decays
__global__ void scan_decay_prod_kernel(Batch b, int nd, int chunk, int nchunks, const float* __restrict__ decay, float* __restrict__ prod) {
    const int sq = blockIdx.x / nchunks, c = blockIdx.x - sq * nchunks, k = blockIdx.y * blockDim.x + threadIdx.x;
    const int len = b.seq_len[sq], start = b.seq_start[sq];
    if (k >= nd || c * chunk >= len) return;
    const int t1 = len - c * chunk < chunk ? len - c * chunk : chunk;
    const float* p = decay + (size_t)(start + c * chunk) * nd + k;
    float pr = 1.f;
#pragma unroll 8
    for (int t = 0; t < t1; ++t) pr *= p[(size_t)t * nd];
    prod[(size_t)(start / chunk + sq + c) * nd + k] = pr;
}

__device__ __forceinline__ float gla_decay_of(float z, float inv_tau) {        // sigmoid(z)^(1 / tau); ln sigmoid(z) = min(z, 0) - ln(1 + exp(-|z|))
    return expf((fminf(z, 0.f) - log1pf(expf(-fabsf(z)))) * inv_tau);
}

// The same on tensor cores (bf16 storage): 64 tokens x 64 channels per block, a warp per 16 tokens.  The float low-rank rows enter as a
// two-term bf16 split, so that the product sees them to 2^-17; a2 is bf16 as stored.  rp: rank rounded up to 16.
constexpr int GM_TOK = 64, GM_CH = 64;
__global__ void __launch_bounds__(128) gla_decay_mma_kernel(int n, int rank, int rp, int nout, const float* __restrict__ a1, int ld, const __nv_bfloat16* __restrict__ a2,
                                                            const __nv_bfloat16* __restrict__ bias, float inv_tau, float* __restrict__ decay) {
    extern __shared__ __align__(16) unsigned char gm_raw[];
    __shared__ float zb[GM_CH];
    const int S = rp + 8, i0 = blockIdx.x * GM_TOK, c0 = blockIdx.y * GM_CH;
    __nv_bfloat16* Ah = reinterpret_cast<__nv_bfloat16*>(gm_raw);
    __nv_bfloat16* Al = Ah + GM_TOK * S;
    __nv_bfloat16* B = Al + GM_TOK * S;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5, g4 = lane >> 2, t4 = lane & 3, mi = lane >> 3, rr = lane & 7;
    if (tid < GM_CH) zb[tid] = c0 + tid < nout ? __bfloat162float(bias[c0 + tid]) : 0.f;
    for (int e = tid; e < GM_CH * (rp / 8); e += 128) {       // 16 bytes at a time (rank is a multiple of 8)
        const int c = e / (rp / 8), r = (e - c * (rp / 8)) * 8;
        const bool ok = c0 + c < nout && r < rank;
        am_cp16(smem_u32(B + c * S + r), ok ? a2 + (size_t)(c0 + c) * rank + r : a2, ok);
    }
    am_commit();
    for (int r = lane; r < rp; r += 32) {
        float v[GM_TOK / 4];                                  // independent loads: all in flight at once
#pragma unroll
        for (int k = 0; k < GM_TOK / 4; ++k) { const int t = i0 + warp + 4 * k; v[k] = t < n && r < rank ? a1[(size_t)t * ld + r] : 0.f; }
#pragma unroll
        for (int k = 0; k < GM_TOK / 4; ++k) {
            const int at = (warp + 4 * k) * S + r;
            const __nv_bfloat16 hi = __float2bfloat16_rn(v[k]);
            Ah[at] = hi;
            Al[at] = __float2bfloat16_rn(v[k] - __bfloat162float(hi));
        }
    }
    am_wait<0>();
    __syncthreads();
    if (i0 + warp * 16 >= n) return;
    float acc[GM_CH / 8][4];
#pragma unroll
    for (int j = 0; j < GM_CH / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    const uint32_t ah = smem_u32(Ah), al = smem_u32(Al), bb = smem_u32(B);
    for (int k = 0; k < rp; k += 16) {
        uint32_t fh[4], fl[4];
        const uint32_t at = (uint32_t)((warp * 16 + (lane & 15)) * S + k + (lane >> 4) * 8) * 2u;
        am_ldsm_x4(fh, ah + at);
        am_ldsm_x4(fl, al + at);
#pragma unroll
        for (int jp = 0; jp < GM_CH / 16; ++jp) {
            uint32_t f[4];
            am_ldsm_x4(f, bb + (uint32_t)((jp * 16 + (mi >> 1) * 8 + rr) * S + k + (mi & 1) * 8) * 2u);
            am_mma(acc[2 * jp], fh, f[0], f[1]);
            am_mma(acc[2 * jp + 1], fh, f[2], f[3]);
            am_mma(acc[2 * jp], fl, f[0], f[1]);
            am_mma(acc[2 * jp + 1], fl, f[2], f[3]);
        }
    }
    // every value is finished before the first is stored: the special functions of independent values overlap
#pragma unroll
    for (int j = 0; j < GM_CH / 8; ++j)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[j][e] = gla_decay_of(acc[j][e] + zb[j * 8 + 2 * t4 + (e & 1)], inv_tau);
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        const int i = i0 + warp * 16 + g4 + 8 * k;
        if (i >= n) continue;
        float* row = decay + (size_t)i * nout + c0 + 2 * t4;
#pragma unroll
        for (int j = 0; j < GM_CH / 8; ++j) {
            const int c = c0 + j * 8 + 2 * t4;
            if ((nout & 1) == 0 && c < nout) *reinterpret_cast<float2*>(row + j * 8) = make_float2(acc[j][2 * k], acc[j][2 * k + 1]);
            else { if (c < nout) row[j * 8] = acc[j][2 * k]; if (c + 1 < nout) row[j * 8 + 1] = acc[j][2 * k + 1]; }
        }
    }
}

// decay of gated linear attention: a thread owns one output channel and GD_TOK tokens; the tokens' low-rank rows lie in shared memory
constexpr int GD_TOK = 8, GD_THREADS = 128;
template <typename T>
__global__ void __launch_bounds__(GD_THREADS) gla_decay_kernel(int n, int rank, int nout, const float* __restrict__ a1, int ld, const T* __restrict__ a2,
                                                               const T* __restrict__ bias, float inv_tau, float* __restrict__ decay) {
    extern __shared__ float rows[];                  // [rank][GD_TOK]
    const int i0 = blockIdx.x * GD_TOK, c = blockIdx.y * GD_THREADS + threadIdx.x;
    for (int idx = threadIdx.x; idx < rank * GD_TOK; idx += GD_THREADS) {
        const int t = idx / rank, r = idx - t * rank;
        rows[r * GD_TOK + t] = i0 + t < n ? a1[(size_t)(i0 + t) * ld + r] : 0.f;
    }
    __syncthreads();
    if (c >= nout) return;
    float acc[GD_TOK];
    const float bz = to_f(bias[c]);
#pragma unroll
    for (int t = 0; t < GD_TOK; ++t) acc[t] = bz;
    const T* wr = a2 + (size_t)c * rank;
#pragma unroll 4
    for (int r = 0; r < rank; ++r) {
        const float w = to_f(wr[r]);
#pragma unroll
        for (int t = 0; t < GD_TOK; ++t) acc[t] = fmaf(w, rows[r * GD_TOK + t], acc[t]);
    }
#pragma unroll
    for (int t = 0; t < GD_TOK; ++t)
        if (i0 + t < n) decay[(size_t)(i0 + t) * nout + c] = gla_decay_of(acc[t], inv_tau);
}

template <typename T>
__global__ void delta_post_kernel(DeltaDims D, const float* __restrict__ o, const T* __restrict__ w, float eps, const float* __restrict__ g, int ldg,
                                  T* __restrict__ y, int act) {
    const int i = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = blockDim.x >> 5;
    for (int h = blockIdx.y * nw + warp; h < D.H; h += gridDim.y * nw) {
        const float* x = o + ((size_t)i * D.H + h) * D.dv;
        float ss = 0.f;
        for (int c = lane; c < D.dv; c += 32) ss += x[c] * x[c];
        ss = warp_sum(ss);
        const float inv = 1.f / sqrtf(ss / (float)D.dv + eps);
        for (int c = lane; c < D.dv; c += 32) {
            const float z = g[(size_t)i * ldg + (size_t)h * D.dv + c];
            y[((size_t)i * D.H + h) * D.dv + c] = from_f<T>(x[c] * inv * to_f(w[c]) * (act ? sigmoid_f(z) : silu_f(z)));
        }
    }
}

}  // namespace

int launch_delta_prep(int dt, const DeltaDims& D, int n, float* qkv, int ld, const float* a_raw, int lda, const float* b_raw, int ldb_,
                      const void* A_log, const void* dt_bias, float* beta, float* decay, cudaStream_t s) {
    if (n <= 0) return WF_OK;
    if (D.Hk <= 0 || D.H % D.Hk) { set_error("delta: %d heads over %d key heads", D.H, D.Hk); return WF_ERR_INVALID; }
    if (dt == WF_BF16) delta_prep_kernel<<<n, 128, 0, s>>>(D, qkv, ld, a_raw, lda, b_raw, ldb_, (const __nv_bfloat16*)A_log, (const __nv_bfloat16*)dt_bias, beta, decay);
    else delta_prep_kernel<<<n, 128, 0, s>>>(D, qkv, ld, a_raw, lda, b_raw, ldb_, (const float*)A_log, (const float*)dt_bias, beta, decay);
    return launch_check(cudaGetLastError(), "delta_prep");
}

namespace {
template <bool VEC, bool DELTA>
int delta_rule_launch(const Batch& b, const DeltaDims& D, const float* qkv, int ld, const float* beta, const float* decay, float* state,
                      size_t slot_stride, float* o, cudaStream_t s, ScanArgs sa = ScanArgs()) {
    const bool decode = b.n == b.nseq;                     // every sequence brings one token
    // two columns per thread where a block's 32 columns exist and the chunks in parallel still fill the machine
    const bool wide = !DELTA && sa.pass && D.d <= 128 && D.dv + D.ones_col >= 32 && (long long)b.nseq * sa.nchunks * D.H * ((D.dv + D.ones_col + 31) / 32) >= 4 * sm_count();
    const int parts = decode ? 4 : 8, cols = DR_THREADS / parts * (wide ? 2 : 1);
    dim3 grid(sa.pass ? b.nseq * sa.nchunks : b.nseq, D.H, (D.dv + D.ones_col + cols - 1) / cols);
    const int dpt_raw = (D.d + parts - 1) / parts, dpt_t = dpt_raw <= 8 ? 8 : (dpt_raw <= 16 ? 16 : (dpt_raw <= 32 ? 32 : 64));
    const size_t smem = 2 * ((size_t)(VEC ? 3 : 2) * DR_TT * parts * (dpt_t + 4) + DR_TT * cols + 2 * DR_TT) * sizeof(float);   // two token groups, padded rows
    static DevOnce once;
    if (once.need()) {
#define DR_ATTR(dp, pa) cudaFuncSetAttribute(delta_rule_kernel<dp, pa, VEC, DELTA, 1>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024)
        DR_ATTR(8, 8); DR_ATTR(16, 8); DR_ATTR(32, 8); DR_ATTR(64, 8); DR_ATTR(8, 4); DR_ATTR(16, 4); DR_ATTR(32, 4); DR_ATTR(64, 4);
#undef DR_ATTR
        if (!DELTA) {
            cudaFuncSetAttribute(delta_rule_kernel<8, 8, VEC, DELTA, DELTA ? 1 : 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
            cudaFuncSetAttribute(delta_rule_kernel<16, 8, VEC, DELTA, DELTA ? 1 : 2>, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
        }
    }
    const int dpt = (D.d + parts - 1) / parts;
    {   // 16-byte staging copies when every row the kernel stages starts aligned and has a multiple of 4 entries
        const int qo = D.q_off >= 0 ? D.q_off : 0, ko = D.k_off >= 0 ? D.k_off : D.Hk * D.d, vo = D.v_off >= 0 ? D.v_off : 2 * D.Hk * D.d;
        sa.v4 = D.d % 4 == 0 && D.dv % 4 == 0 && ld % 4 == 0 && qo % 4 == 0 && ko % 4 == 0 && vo % 4 == 0 && ((uintptr_t)qkv & 15) == 0 && ((uintptr_t)decay & 15) == 0;
    }
#define DR_LAUNCH(dp, pa, nc) delta_rule_kernel<dp, pa, VEC, DELTA, nc><<<grid, DR_THREADS, smem, s>>>(b, D, qkv, ld, beta, decay, state, slot_stride, o, sa)
    if (D.d > 256 || smem > 160 * 1024) { set_error("delta: key dimension %d above the supported 256", D.d); return WF_ERR_UNSUPPORTED; }
    if (wide) { if (dpt <= 8) DR_LAUNCH(8, 8, (DELTA ? 1 : 2)); else DR_LAUNCH(16, 8, (DELTA ? 1 : 2)); }
    else if (decode) { if (dpt <= 8) DR_LAUNCH(8, 4, 1); else if (dpt <= 16) DR_LAUNCH(16, 4, 1); else if (dpt <= 32) DR_LAUNCH(32, 4, 1); else DR_LAUNCH(64, 4, 1); }
    else { if (dpt <= 8) DR_LAUNCH(8, 8, 1); else if (dpt <= 16) DR_LAUNCH(16, 8, 1); else if (dpt <= 32) DR_LAUNCH(32, 8, 1); else DR_LAUNCH(64, 8, 1); }
#undef DR_LAUNCH
    return launch_check(cudaGetLastError(), "delta_rule");
}
}  // namespace

int launch_delta_rule(const Batch& b, const DeltaDims& D, const float* qkv, int ld, const float* beta, const float* decay, float* state,
                      size_t slot_stride, float* o, cudaStream_t s, const ScanWorkspace* scan) {
    if (b.nseq <= 0) return WF_OK;
    if (D.Hk <= 0 || D.H % D.Hk) { set_error("delta: %d heads over %d key heads", D.H, D.Hk); return WF_ERR_INVALID; }
    if (D.ones_col && !D.no_delta) { set_error("delta: the all-ones column belongs to the plain recurrence"); return WF_ERR_UNSUPPORTED; }
    if (D.no_delta) {
        auto plain = [&](const ScanArgs& sa) {
            return D.vec_decay ? delta_rule_launch<true, false>(b, D, qkv, ld, beta, decay, state, slot_stride, o, s, sa)
                               : delta_rule_launch<false, false>(b, D, qkv, ld, beta, decay, state, slot_stride, o, s, sa);
        };
        // long portions: chunks in parallel (two short sequential passes instead of one long one)
        if (scan && scan->local && b.n != b.nseq && b.max_len >= 2 * SCAN_CHUNK && b.n / SCAN_CHUNK + b.nseq + 1 <= scan->chunks) {
            ScanArgs sa;
            sa.chunk = SCAN_CHUNK; sa.nchunks = (b.max_len + SCAN_CHUNK - 1) / SCAN_CHUNK;
            sa.local = scan->local; sa.start = scan->start; sa.prod = scan->prod;
            sa.pass = 1;
            if (int rc = plain(sa)) return rc;
            if (D.vec_decay) {
                const int nd = D.H * D.d;
                scan_decay_prod_kernel<<<dim3(b.nseq * sa.nchunks, (nd + 127) / 128), 128, 0, s>>>(b, nd, SCAN_CHUNK, sa.nchunks, decay, scan->prod);
                if (int rc = launch_check(cudaGetLastError(), "scan_decay_prod")) return rc;
            }
            const int dd = D.d * (D.dv + D.ones_col);
            scan_prefix_kernel<<<dim3(b.nseq, D.H, (dd + 255) / 256), 256, 0, s>>>(b, D.H, dd, SCAN_CHUNK, state, slot_stride, scan->local, scan->start, scan->prod, D.vec_decay ? D.d : 0);
            if (int rc = launch_check(cudaGetLastError(), "scan_prefix")) return rc;
            sa.pass = 3;
            return plain(sa);
        }
        return plain(ScanArgs());
    }
    return D.vec_decay ? delta_rule_launch<true, true>(b, D, qkv, ld, beta, decay, state, slot_stride, o, s)
                       : delta_rule_launch<false, true>(b, D, qkv, ld, beta, decay, state, slot_stride, o, s);
}

int launch_delta_post(int dt, const DeltaDims& D, int n, const float* o, const void* w, float eps, const float* g, int ldg, void* y, cudaStream_t s, int act) {
    if (n <= 0) return WF_OK;
    const dim3 grid(n, n < 64 ? (D.H + 3) / 4 : 1);
    if (dt == WF_BF16) delta_post_kernel<<<grid, 128, 0, s>>>(D, o, (const __nv_bfloat16*)w, eps, g, ldg, (__nv_bfloat16*)y, act);
    else delta_post_kernel<<<grid, 128, 0, s>>>(D, o, (const float*)w, eps, g, ldg, (float*)y, act);
    return launch_check(cudaGetLastError(), "delta_post");
}

int launch_gla_decay(int dt, int n, int rank, int nout, const float* a1, int ld, const void* a2, const void* bias, float tau, float* decay, cudaStream_t s) {
    if (n <= 0) return WF_OK;
    const int rp = (rank + 15) / 16 * 16;
    const size_t mma_smem = (size_t)(2 * GM_TOK + GM_CH) * (rp + 8) * 2;
    if (dt == WF_BF16 && rank > 0 && tau > 0.f && rank % 8 == 0 && mma_smem <= 160 * 1024) {
        static DevOnce once;
        if (once.need()) cudaFuncSetAttribute(gla_decay_mma_kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, 160 * 1024);
        gla_decay_mma_kernel<<<dim3((n + GM_TOK - 1) / GM_TOK, (nout + GM_CH - 1) / GM_CH), 128, mma_smem, s>>>(n, rank, rp, nout, a1, ld, (const __nv_bfloat16*)a2,
                                                                                                              (const __nv_bfloat16*)bias, 1.f / tau, decay);
        return launch_check(cudaGetLastError(), "gla_decay_mma");
    }
    const size_t smem = (size_t)rank * GD_TOK * sizeof(float);
    if (rank <= 0 || !(tau > 0.f) || smem > 48 * 1024) { set_error("gla: decay projection of rank %d, tau %g", rank, tau); return WF_ERR_UNSUPPORTED; }
    const dim3 grid((n + GD_TOK - 1) / GD_TOK, (nout + GD_THREADS - 1) / GD_THREADS);
    if (dt == WF_BF16) gla_decay_kernel<<<grid, GD_THREADS, smem, s>>>(n, rank, nout, a1, ld, (const __nv_bfloat16*)a2, (const __nv_bfloat16*)bias, 1.f / tau, decay);
    else gla_decay_kernel<<<grid, GD_THREADS, smem, s>>>(n, rank, nout, a1, ld, (const float*)a2, (const float*)bias, 1.f / tau, decay);
    return launch_check(cudaGetLastError(), "gla_decay");
}

int launch_ssd_prep(int dt, int n, int H, const float* dt_raw, int ld, const void* A_log, const void* dt_bias, float* step, float* decay, cudaStream_t s) {
    if (n <= 0) return WF_OK;
    const int blocks = (n * H + 127) / 128;
    if (dt == WF_BF16) ssd_prep_kernel<<<blocks, 128, 0, s>>>(n, H, dt_raw, ld, (const __nv_bfloat16*)A_log, (const __nv_bfloat16*)dt_bias, step, decay);
    else ssd_prep_kernel<<<blocks, 128, 0, s>>>(n, H, dt_raw, ld, (const float*)A_log, (const float*)dt_bias, step, decay);
    return launch_check(cudaGetLastError(), "ssd_prep");
}

int launch_ssd_post(int dt, int n, int H, int dv, int groups, const float* o, const float* x, int ldx, const float* z, int ldz, const void* Dskip,
                    const void* w, float eps, void* y, cudaStream_t s) {
    if (n <= 0) return WF_OK;
    if (groups <= 0 || (H * dv) % groups) { set_error("ssd: %d channels not divisible into %d norm groups", H * dv, groups); return WF_ERR_INVALID; }
    const int gw = H * dv / groups;
    const int threads = gw >= 1024 ? 256 : (gw >= 256 ? 128 : 64);
    const dim3 grid(n, groups);
    if (dt == WF_BF16) ssd_post_kernel<<<grid, threads, 0, s>>>(H, dv, groups, o, x, ldx, z, ldz, (const __nv_bfloat16*)Dskip, (const __nv_bfloat16*)w, eps, (__nv_bfloat16*)y);
    else ssd_post_kernel<<<grid, threads, 0, s>>>(H, dv, groups, o, x, ldx, z, ldz, (const float*)Dskip, (const float*)w, eps, (float*)y);
    return launch_check(cudaGetLastError(), "ssd_post");
}

}  // namespace seq
}  // namespace wf
