// Row-wise kernels of the sequence models: embedding gather, grouped RMS norm (+ residual add), element-wise norms with everything that lies
// between two sublayers, causal depthwise taps with carried state.
#include "seq_kernels.cuh"

namespace wf {
namespace seq {

template <typename T>
__global__ void embed_f32_kernel(const T* __restrict__ table, const int32_t* __restrict__ tokens, int W, float* __restrict__ x, float scale, T* __restrict__ x_t,
                                 const T* __restrict__ pos_table, const int32_t* __restrict__ tok_pos) {
    const int i = blockIdx.x;
    const T* row = table + (size_t)tokens[i] * W;
    const T* prow = pos_table ? pos_table + (size_t)tok_pos[i] * W : nullptr;
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
        float v = to_f(row[c]) * scale;
        if (prow) v += to_f(prow[c]);
        x[(size_t)i * W + c] = v;
        if (x_t) x_t[(size_t)i * W + c] = from_f<T>(v);
    }
}

int launch_embed_f32(int dt, const void* table, const int32_t* tokens, int n, int W, float* x, cudaStream_t s, float scale, void* x_t,
                     const void* pos_table, const int32_t* tok_pos) {
    if (n <= 0) return WF_OK;
    if (dt == WF_BF16) embed_f32_kernel<<<n, 256, 0, s>>>((const __nv_bfloat16*)table, tokens, W, x, scale, (__nv_bfloat16*)x_t, (const __nv_bfloat16*)pos_table, tok_pos);
    else embed_f32_kernel<<<n, 256, 0, s>>>((const float*)table, tokens, W, x, scale, (float*)x_t, (const float*)pos_table, tok_pos);
    return launch_check(cudaGetLastError(), "embed_f32");
}

__global__ void axpby_kernel(float* __restrict__ y, float a, const float* __restrict__ y2, float b, size_t count) {
    for (size_t k = (size_t)blockIdx.x * blockDim.x + threadIdx.x; k < count; k += (size_t)gridDim.x * blockDim.x) y[k] = a * y[k] + b * y2[k];
}

int launch_axpby(float* y, float a, const float* y2, float b, size_t count, cudaStream_t s) {
    if (count == 0) return WF_OK;
    const int blocks = (int)((count + 255) / 256 > 4096 ? 4096 : (count + 255) / 256);
    axpby_kernel<<<blocks, 256, 0, s>>>(y, a, y2, b, count);
    return launch_check(cudaGetLastError(), "axpby");
}

// x[i, :] = table[tokens[i], :] + position vector of tok_pos[i]: entry 2k = sin(a), entry 2k + 1 = cos(a), a = pos * base^(-2k / W).
// The frequency and the angle are formed in double so that the float result is the correctly rounded one also at large positions.
template <typename T>
__global__ void embed_pos_kernel(const T* __restrict__ table, const int32_t* __restrict__ tokens, const int32_t* __restrict__ tok_pos, int W, float base,
                                 float* __restrict__ x, T* __restrict__ x_t) {
    const int i = blockIdx.x;
    const T* row = table + (size_t)tokens[i] * W;
    const double pos = (double)tok_pos[i], lb = log2((double)base);
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
        const double a = pos * exp2(-2.0 * (double)(c >> 1) / (double)W * lb);
        const float v = to_f(row[c]) + (float)((c & 1) ? cos(a) : sin(a));
        x[(size_t)i * W + c] = v;
        if (x_t) x_t[(size_t)i * W + c] = from_f<T>(v);
    }
}

int launch_embed_pos(int dt, const void* table, const int32_t* tokens, const int32_t* tok_pos, int n, int W, float base, float* x, void* x_t, cudaStream_t s) {
    if (n <= 0) return WF_OK;
    if (dt == WF_BF16) embed_pos_kernel<<<n, 256, 0, s>>>((const __nv_bfloat16*)table, tokens, tok_pos, W, base, x, (__nv_bfloat16*)x_t);
    else embed_pos_kernel<<<n, 256, 0, s>>>((const float*)table, tokens, tok_pos, W, base, x, (float*)x_t);
    return launch_check(cudaGetLastError(), "embed_pos");
}

// x_t[i, :] = T(x[i, :])
template <typename T>
__global__ void round_rows_kernel(const float* __restrict__ x, size_t count, T* __restrict__ x_t) {
    for (size_t k = (size_t)blockIdx.x * blockDim.x + threadIdx.x; k < count; k += (size_t)gridDim.x * blockDim.x) x_t[k] = from_f<T>(x[k]);
}

int launch_round_rows(int dt, const float* x, int n, int W, void* x_t, cudaStream_t s) {
    if (n <= 0) return WF_OK;
    const size_t count = (size_t)n * W;
    const int blocks = (int)((count + 255) / 256 > 4096 ? 4096 : (count + 255) / 256);
    if (dt == WF_BF16) round_rows_kernel<<<blocks, 256, 0, s>>>(x, count, (__nv_bfloat16*)x_t);
    else round_rows_kernel<<<blocks, 256, 0, s>>>(x, count, (float*)x_t);
    return launch_check(cudaGetLastError(), "round_rows");
}

// RMS norm with ONE gain: v = mult * gain * (y + bias) / sqrt(mean((y + bias)^2) + eps) [+ res].  One block per row; the row is kept in
// registers between the two passes (up to SN_PER values per thread, re-read beyond that).
constexpr int SN_THREADS = 256, SN_PER = 8;
template <typename T>
__global__ void __launch_bounds__(SN_THREADS) scalar_rmsnorm_kernel(const float* __restrict__ y, int ldy, const T* __restrict__ bias, const T* __restrict__ gain, float mult,
                                                                    float eps, int W, const float* res, float* out, int ldo, T* __restrict__ out_t, int ldt,
                                                                    const int32_t* __restrict__ rows) {
    __shared__ float scratch[33];
    const int i = blockIdx.x;
    const int src = rows ? rows[i] : i;
    const float* yr = y + (size_t)src * ldy;
    float v[SN_PER];
    float ss = 0.f;
#pragma unroll
    for (int t = 0; t < SN_PER; ++t) {
        const int c = threadIdx.x + t * SN_THREADS;
        v[t] = c < W ? yr[c] + (bias ? to_f(bias[c]) : 0.f) : 0.f;
        ss = fmaf(v[t], v[t], ss);
    }
    for (int c = threadIdx.x + SN_PER * SN_THREADS; c < W; c += SN_THREADS) { const float u = yr[c] + (bias ? to_f(bias[c]) : 0.f); ss = fmaf(u, u, ss); }
    ss = block_sum(ss, scratch);
    const float k = mult * to_f(gain[0]) / sqrtf(ss / (float)W + eps);
#pragma unroll
    for (int t = 0; t < SN_PER; ++t) {
        const int c = threadIdx.x + t * SN_THREADS;
        if (c < W) {
            float u = v[t] * k;
            if (res) u += res[(size_t)src * ldo + c];
            if (out) out[(size_t)i * ldo + c] = u;
            if (out_t) out_t[(size_t)i * ldt + c] = from_f<T>(u);
        }
    }
    for (int c = threadIdx.x + SN_PER * SN_THREADS; c < W; c += SN_THREADS) {
        float u = (yr[c] + (bias ? to_f(bias[c]) : 0.f)) * k;
        if (res) u += res[(size_t)src * ldo + c];
        if (out) out[(size_t)i * ldo + c] = u;
        if (out_t) out_t[(size_t)i * ldt + c] = from_f<T>(u);
    }
}

int launch_scalar_rmsnorm(int dt, const float* y, int ldy, const void* bias, const void* gain, float mult, float eps, int n, int W, const float* res, float* out,
                          int ldo, void* out_t, int ldt, const int32_t* rows, cudaStream_t s) {
    if (n <= 0) return WF_OK;
    if (res && rows && out == res) { set_error("scalar_rmsnorm: gathered rows cannot be added in place"); return WF_ERR_INVALID; }
    if (dt == WF_BF16) scalar_rmsnorm_kernel<<<n, SN_THREADS, 0, s>>>(y, ldy, (const __nv_bfloat16*)bias, (const __nv_bfloat16*)gain, mult, eps, W, res, out, ldo, (__nv_bfloat16*)out_t, ldt, rows);
    else scalar_rmsnorm_kernel<<<n, SN_THREADS, 0, s>>>(y, ldy, (const float*)bias, (const float*)gain, mult, eps, W, res, out, ldo, (float*)out_t, ldt, rows);
    return launch_check(cudaGetLastError(), "scalar_rmsnorm");
}

// y[i, :] += bias
template <typename T>
__global__ void add_bias_kernel(float* __restrict__ y, int ld, const T* __restrict__ bias, int W) {
    for (int c = threadIdx.x; c < W; c += blockDim.x) y[(size_t)blockIdx.x * ld + c] += to_f(bias[c]);
}

int launch_add_bias(int dt, float* y, int ld, const void* bias, int n, int W, cudaStream_t s) {
    if (n <= 0 || !bias) return WF_OK;
    if (dt == WF_BF16) add_bias_kernel<<<n, 256, 0, s>>>(y, ld, (const __nv_bfloat16*)bias, W);
    else add_bias_kernel<<<n, 256, 0, s>>>(y, ld, (const float*)bias, W);
    return launch_check(cudaGetLastError(), "add_bias");
}

// one block per (row, group).  x2 (optional): the normalised quantity is a * x + b * x2 (two mixers' outputs combined on the way in)
template <typename T>
__global__ void group_rmsnorm_kernel(const float* __restrict__ x, int ldx, const T* __restrict__ w, int gw, float eps, const float* res,
                                     float* y, int ldy, T* __restrict__ y_t, int ldt, const int32_t* __restrict__ rows, const float* __restrict__ x2, float a,
                                     float b, float w_offset) {
    __shared__ float scratch[33];
    const int i = blockIdx.x, g = blockIdx.y;
    const int src = rows ? rows[i] : i;
    const float* xr = x + (size_t)src * ldx + (size_t)g * gw;
    const float* xr2 = x2 ? x2 + (size_t)src * ldx + (size_t)g * gw : nullptr;
    float ss = 0.f;
    for (int c = threadIdx.x; c < gw; c += blockDim.x) { const float v = xr2 ? a * xr[c] + b * xr2[c] : xr[c]; ss += v * v; }
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)gw + eps);
    for (int c = threadIdx.x; c < gw; c += blockDim.x) {
        float v = (xr2 ? a * xr[c] + b * xr2[c] : xr[c]) * inv * (w_offset + to_f(w[g * gw + c]));
        if (res) v += res[(size_t)src * ldy + g * gw + c];
        if (y) y[(size_t)i * ldy + g * gw + c] = v;
        if (y_t) y_t[(size_t)i * ldt + g * gw + c] = from_f<T>(v);
    }
}

int launch_group_rmsnorm(int dt, const float* x, int ldx, const void* w, int groups, float eps, int n, int W, const float* res, float* y,
                         int ldy, void* y_t, int ldt, const int32_t* rows, cudaStream_t s, const float* x2, float a, float b, float w_offset) {
    if (n <= 0) return WF_OK;
    if (groups <= 0 || W % groups) { set_error("group_rmsnorm: width %d not divisible into %d groups", W, groups); return WF_ERR_INVALID; }
    if (res && rows && y == res) { set_error("group_rmsnorm: gathered rows cannot be added in place"); return WF_ERR_INVALID; }
    const int gw = W / groups;
    const int threads = gw >= 2048 ? 512 : (gw >= 1024 ? 256 : (gw >= 256 ? 128 : 64));
    dim3 grid(n, groups);
    if (dt == WF_BF16) group_rmsnorm_kernel<<<grid, threads, 0, s>>>(x, ldx, (const __nv_bfloat16*)w, gw, eps, res, y, ldy, (__nv_bfloat16*)y_t, ldt, rows, x2, a, b, w_offset);
    else group_rmsnorm_kernel<<<grid, threads, 0, s>>>(x, ldx, (const float*)w, gw, eps, res, y, ldy, (float*)y_t, ldt, rows, x2, a, b, w_offset);
    return launch_check(cudaGetLastError(), "group_rmsnorm");
}

// One block per row; the updated row stays in registers between the sum of squares and the two scaled copies (up to AD_PER elements per
// thread; wider rows are re-read from x, which the same thread has just written).
constexpr int AD_THREADS = 256, AD_PER = 8;
template <typename T>
__global__ void __launch_bounds__(AD_THREADS) add_dual_norm_kernel(float* __restrict__ x, const float* __restrict__ y1, float a1, const float* __restrict__ y2, float a2,
                                                                     const float* __restrict__ y3, const T* __restrict__ w1, const T* __restrict__ w2, float w_offset,
                                                                     float eps, int W, T* __restrict__ h1, T* __restrict__ h2) {
    __shared__ float scratch[33];
    const size_t base = (size_t)blockIdx.x * W;
    const bool adds = y1 || y2 || y3;
    float keep[AD_PER];
    float ss = 0.f;
    int k = 0;
    for (int c = threadIdx.x; c < W; c += AD_THREADS, ++k) {
        float v = x[base + c];
        if (adds) {
            float t = 0.f;
            if (y1) t = a1 * y1[base + c];
            if (y2) t = fmaf(a2, y2[base + c], t);
            if (y3) t += y3[base + c];
            v += t;
            x[base + c] = v;
        }
        if (k < AD_PER) keep[k] = v;
        ss = fmaf(v, v, ss);
    }
    if (!w1 && !w2) return;
    ss = block_sum(ss, scratch);
    const float inv = 1.f / sqrtf(ss / (float)W + eps);
    k = 0;
    for (int c = threadIdx.x; c < W; c += AD_THREADS, ++k) {
        const float r = (k < AD_PER ? keep[k] : x[base + c]) * inv;
        if (w1) h1[base + c] = from_f<T>(r * (w_offset + to_f(w1[c])));
        if (w2) h2[base + c] = from_f<T>(r * (w_offset + to_f(w2[c])));
    }
}

int launch_add_dual_norm(int dt, float* x, const float* y1, float a1, const float* y2, float a2, const float* y3, const void* w1, const void* w2,
                         float w_offset, float eps, int n, int W, void* h1, void* h2, cudaStream_t s) {
    if (n <= 0) return WF_OK;
    if (dt == WF_BF16) add_dual_norm_kernel<<<n, AD_THREADS, 0, s>>>(x, y1, a1, y2, a2, y3, (const __nv_bfloat16*)w1, (const __nv_bfloat16*)w2, w_offset, eps, W, (__nv_bfloat16*)h1, (__nv_bfloat16*)h2);
    else add_dual_norm_kernel<<<n, AD_THREADS, 0, s>>>(x, y1, a1, y2, a2, y3, (const float*)w1, (const float*)w2, w_offset, eps, W, (float*)h1, (float*)h2);
    return launch_check(cudaGetLastError(), "add_dual_norm");
}

// sum over the block of the squared distances from the mean, the row's values in keep (up to PER per thread) and in row (read beyond those)
template <int PER>
__device__ __forceinline__ float block_sq_dev(const float (&keep)[PER], const float* row, int W, float mean, float* scratch) {
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < PER; ++k) {
        const int c = threadIdx.x + k * blockDim.x;
        if (c < W) { const float d = keep[k] - mean; ss = fmaf(d, d, ss); }
    }
    for (int c = threadIdx.x + PER * blockDim.x; c < W; c += blockDim.x) { const float d = row[c] - mean; ss = fmaf(d, d, ss); }
    return block_sum(ss, scratch);
}

// one block per row; the row stays in registers between the two statistics and the store (re-read beyond LN_PER values per thread)
constexpr int LN_PER = 8;
template <typename T>
__global__ void __launch_bounds__(512) layer_norm_kernel(const float* __restrict__ x, int ldx, const T* __restrict__ w, const T* __restrict__ b, float eps, int W,
                                                         float* __restrict__ y, int ldy, T* __restrict__ y_t, int ldt, const int32_t* __restrict__ rows) {
    __shared__ float scratch[33];
    const int i = blockIdx.x;
    const float* row = x + (size_t)(rows ? rows[i] : i) * ldx;
    float keep[LN_PER], sum = 0.f;
#pragma unroll
    for (int k = 0; k < LN_PER; ++k) {
        const int c = threadIdx.x + k * blockDim.x;
        keep[k] = c < W ? row[c] : 0.f;
        sum += keep[k];
    }
    for (int c = threadIdx.x + LN_PER * blockDim.x; c < W; c += blockDim.x) sum += row[c];
    const float mean = block_sum(sum, scratch) / (float)W;
    const float inv = 1.f / sqrtf(block_sq_dev(keep, row, W, mean, scratch) / (float)W + eps);
#pragma unroll
    for (int k = 0; k < LN_PER; ++k) {
        const int c = threadIdx.x + k * blockDim.x;
        if (c >= W) continue;
        const float v = (keep[k] - mean) * inv * to_f(w[c]) + to_f(b[c]);
        if (y) y[(size_t)i * ldy + c] = v;
        if (y_t) y_t[(size_t)i * ldt + c] = from_f<T>(v);
    }
    for (int c = threadIdx.x + LN_PER * blockDim.x; c < W; c += blockDim.x) {
        const float v = (row[c] - mean) * inv * to_f(w[c]) + to_f(b[c]);
        if (y) y[(size_t)i * ldy + c] = v;
        if (y_t) y_t[(size_t)i * ldt + c] = from_f<T>(v);
    }
}

int row_threads(int W) { return W > 1024 ? 512 : (W > 256 ? 256 : 128); }

int launch_layer_norm(int dt, const float* x, int ldx, const void* w, const void* b, float eps, int n, int W, float* y, int ldy, void* y_t, int ldt,
                      const int32_t* rows, cudaStream_t s) {
    if (n <= 0) return WF_OK;
    if (dt == WF_BF16) layer_norm_kernel<<<n, row_threads(W), 0, s>>>(x, ldx, (const __nv_bfloat16*)w, (const __nv_bfloat16*)b, eps, W, y, ldy, (__nv_bfloat16*)y_t, ldt, rows);
    else layer_norm_kernel<<<n, row_threads(W), 0, s>>>(x, ldx, (const float*)w, (const float*)b, eps, W, y, ldy, (float*)y_t, ldt, rows);
    return launch_check(cudaGetLastError(), "layer_norm");
}

// one block per row (launch_branch_add_norm)
template <typename T>
__global__ void __launch_bounds__(512) branch_add_norm_kernel(float* __restrict__ x, BranchSum bs, const T* __restrict__ w, const T* __restrict__ b, float w_offset, float eps,
                                                              int W, T* __restrict__ h) {
    __shared__ float scratch[33];
    const size_t base = (size_t)blockIdx.x * W;
    float* row = x + base;
    const float* y1 = bs.y1 ? bs.y1 + base : nullptr;
    const float* y2 = bs.y2 ? bs.y2 + base : nullptr;
    const float* y3 = bs.y3 ? bs.y3 + base : nullptr;
    const float* gate = bs.gate ? bs.gate + (size_t)blockIdx.x * bs.ldg : nullptr;
    const T *pw1 = (const T*)bs.pw1, *pw2 = (const T*)bs.pw2, *gb1 = (const T*)bs.gb1, *gb2 = (const T*)bs.gb2;
    float k1[LN_PER], k2[LN_PER];                  // the pair's outputs stay in registers between their norms and the sum
    float f1 = bs.a1, f2 = bs.a2;
#pragma unroll
    for (int k = 0; k < LN_PER; ++k) {
        const int c = threadIdx.x + k * blockDim.x;
        k1[k] = y1 && c < W ? y1[c] : 0.f;
        k2[k] = y2 && c < W ? y2[c] : 0.f;
    }
    if (pw1 && y1) {
        float s1 = 0.f, s2 = 0.f;
#pragma unroll
        for (int k = 0; k < LN_PER; ++k) { s1 = fmaf(k1[k], k1[k], s1); s2 = fmaf(k2[k], k2[k], s2); }
        for (int c = threadIdx.x + LN_PER * blockDim.x; c < W; c += blockDim.x) { s1 = fmaf(y1[c], y1[c], s1); if (y2) s2 = fmaf(y2[c], y2[c], s2); }
        f1 *= 1.f / sqrtf(block_sum(s1, scratch) / (float)W + eps);
        if (y2) f2 *= 1.f / sqrtf(block_sum(s2, scratch) / (float)W + eps);
    }
    auto updated = [&](int c, float v1, float v2) {
        float v = row[c];
        if (y1) {
            float m = f1 * v1 * (pw1 ? to_f(pw1[c]) : 1.f);
            if (y2) m += f2 * v2 * (pw2 ? to_f(pw2[c]) : 1.f);
            float t = gate ? sigmoid_f(gate[c] + to_f(gb1[c])) * m : m;
            if (y3) t += gate ? sigmoid_f(gate[W + c] + to_f(gb2[c])) * y3[c] : y3[c];
            v += t;
            row[c] = v;
        }
        return v;
    };
    float keep[LN_PER], sum = 0.f;
#pragma unroll
    for (int k = 0; k < LN_PER; ++k) {
        const int c = threadIdx.x + k * blockDim.x;
        keep[k] = c < W ? updated(c, k1[k], k2[k]) : 0.f;
        sum += keep[k];
    }
    for (int c = threadIdx.x + LN_PER * blockDim.x; c < W; c += blockDim.x) sum += updated(c, y1 ? y1[c] : 0.f, y2 ? y2[c] : 0.f);
    if (!w) return;
    const float mean = b ? block_sum(sum, scratch) / (float)W : 0.f;
    const float inv = 1.f / sqrtf(block_sq_dev(keep, row, W, mean, scratch) / (float)W + eps);
#pragma unroll
    for (int k = 0; k < LN_PER; ++k) {
        const int c = threadIdx.x + k * blockDim.x;
        if (c < W) h[base + c] = from_f<T>((keep[k] - mean) * inv * (w_offset + to_f(w[c])) + (b ? to_f(b[c]) : 0.f));
    }
    for (int c = threadIdx.x + LN_PER * blockDim.x; c < W; c += blockDim.x)
        h[base + c] = from_f<T>((row[c] - mean) * inv * (w_offset + to_f(w[c])) + (b ? to_f(b[c]) : 0.f));
}

template <typename T> __device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<__nv_bfloat16>(const __nv_bfloat16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(v.x << 16), __uint_as_float(v.x & 0xffff0000u), __uint_as_float(v.y << 16), __uint_as_float(v.y & 0xffff0000u));
}
__device__ __forceinline__ void store4(float* p, const float (&v)[4]) { *reinterpret_cast<float4*>(p) = make_float4(v[0], v[1], v[2], v[3]); }
__device__ __forceinline__ void store4(__nv_bfloat16* p, const float (&v)[4]) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v[0], v[1]), b = __floats2bfloat162_rn(v[2], v[3]);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}

// The same with four consecutive elements per load, every input of a row requested before the first is used; a thread owns NV groups of four,
// blockDim.x * NV * 4 >= W.
template <typename T, int NV>
__global__ void __launch_bounds__(1024) branch_add_norm_vec_kernel(float* __restrict__ x, BranchSum bs, const T* __restrict__ w, const T* __restrict__ b, float w_offset, float eps,
                                                                   int W, T* __restrict__ h) {
    __shared__ float scratch[33];
    const size_t base = (size_t)blockIdx.x * W;
    const float* gate = bs.gate ? bs.gate + (size_t)blockIdx.x * bs.ldg : nullptr;
    const float4 zero = make_float4(0.f, 0.f, 0.f, 0.f);
    float4 xv[NV], v1[NV], v2[NV], v3[NV], g1[NV], g2[NV];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = (threadIdx.x + k * blockDim.x) * 4;
        const bool in = c < W;
        xv[k] = in ? load4(x + base + c) : zero;
        v1[k] = in && bs.y1 ? load4(bs.y1 + base + c) : zero;
        v2[k] = in && bs.y2 ? load4(bs.y2 + base + c) : zero;
        v3[k] = in && bs.y3 ? load4(bs.y3 + base + c) : zero;
        g1[k] = in && gate ? load4(gate + c) : zero;
        g2[k] = in && gate && bs.y3 ? load4(gate + W + c) : zero;
    }
    float f1 = bs.a1, f2 = bs.a2;
    if (bs.pw1 && bs.y1) {
        float s1 = 0.f, s2 = 0.f;
#pragma unroll
        for (int k = 0; k < NV; ++k) {
            s1 += v1[k].x * v1[k].x + v1[k].y * v1[k].y + v1[k].z * v1[k].z + v1[k].w * v1[k].w;
            s2 += v2[k].x * v2[k].x + v2[k].y * v2[k].y + v2[k].z * v2[k].z + v2[k].w * v2[k].w;
        }
        f1 *= 1.f / sqrtf(block_sum(s1, scratch) / (float)W + eps);
        if (bs.y2) f2 *= 1.f / sqrtf(block_sum(s2, scratch) / (float)W + eps);
    }
    float sum = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = (threadIdx.x + k * blockDim.x) * 4;
        if (c >= W || !bs.y1) { sum += xv[k].x + xv[k].y + xv[k].z + xv[k].w; continue; }
        const float4 one = make_float4(1.f, 1.f, 1.f, 1.f);
        const float4 p1 = bs.pw1 ? load4((const T*)bs.pw1 + c) : one, p2 = bs.pw2 && bs.y2 ? load4((const T*)bs.pw2 + c) : one;
        const float4 b1 = gate ? load4((const T*)bs.gb1 + c) : zero, b2 = gate && bs.y3 ? load4((const T*)bs.gb2 + c) : zero;
        const float a[4] = {v1[k].x * p1.x, v1[k].y * p1.y, v1[k].z * p1.z, v1[k].w * p1.w}, d[4] = {v2[k].x * p2.x, v2[k].y * p2.y, v2[k].z * p2.z, v2[k].w * p2.w};
        const float u[4] = {v3[k].x, v3[k].y, v3[k].z, v3[k].w}, o[4] = {xv[k].x, xv[k].y, xv[k].z, xv[k].w};
        const float z1[4] = {g1[k].x + b1.x, g1[k].y + b1.y, g1[k].z + b1.z, g1[k].w + b1.w}, z2[4] = {g2[k].x + b2.x, g2[k].y + b2.y, g2[k].z + b2.z, g2[k].w + b2.w};
        float r[4];
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const float m = f1 * a[e] + f2 * d[e];
            r[e] = o[e] + (gate ? sigmoid_f(z1[e]) * m + sigmoid_f(z2[e]) * u[e] : m + u[e]);
            sum += r[e];
        }
        store4(x + base + c, r);
        xv[k] = make_float4(r[0], r[1], r[2], r[3]);
    }
    if (!w) return;
    const float mean = b ? block_sum(sum, scratch) / (float)W : 0.f;
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        if ((threadIdx.x + k * blockDim.x) * 4 >= W) continue;
        xv[k].x -= mean; xv[k].y -= mean; xv[k].z -= mean; xv[k].w -= mean;
        ss += xv[k].x * xv[k].x + xv[k].y * xv[k].y + xv[k].z * xv[k].z + xv[k].w * xv[k].w;
    }
    const float inv = 1.f / sqrtf(block_sum(ss, scratch) / (float)W + eps);
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = (threadIdx.x + k * blockDim.x) * 4;
        if (c >= W) continue;
        const float4 wv = load4(w + c), bv = b ? load4(b + c) : zero;
        const float r[4] = {xv[k].x * inv * (w_offset + wv.x) + bv.x, xv[k].y * inv * (w_offset + wv.y) + bv.y, xv[k].z * inv * (w_offset + wv.z) + bv.z,
                            xv[k].w * inv * (w_offset + wv.w) + bv.w};
        store4(h + base + c, r);
    }
}

int launch_branch_add_norm(int dt, float* x, const BranchSum& bs, const void* w, const void* b, float w_offset, float eps, int n, int W, void* h, cudaStream_t s) {
    if (n <= 0) return WF_OK;
    if ((bs.y2 || bs.y3) && !bs.y1) { set_error("branch_add_norm: a second output without a first"); return WF_ERR_INVALID; }
    if (bs.y2 && (bs.pw1 != nullptr) != (bs.pw2 != nullptr)) { set_error("branch_add_norm: both outputs of a pair are normed or none"); return WF_ERR_INVALID; }
    // rows of up to 8192 elements that start 16-byte aligned stay in registers, four elements per load
    if (W % 4 == 0 && W <= 8192 && bs.ldg % 4 == 0 && ((uintptr_t)bs.gate & 15) == 0) {
        const int nv = W <= 1024 ? 1 : 2, threads = (W / 4 + nv * 32 - 1) / (nv * 32) * 32;
#define BA_LAUNCH(T, NV) branch_add_norm_vec_kernel<T, NV><<<n, threads, 0, s>>>(x, bs, (const T*)w, (const T*)b, w_offset, eps, W, (T*)h)
        if (dt == WF_BF16) { if (nv == 1) BA_LAUNCH(__nv_bfloat16, 1); else BA_LAUNCH(__nv_bfloat16, 2); }
        else { if (nv == 1) BA_LAUNCH(float, 1); else BA_LAUNCH(float, 2); }
#undef BA_LAUNCH
        return launch_check(cudaGetLastError(), "branch_add_norm_vec");
    }
    if (dt == WF_BF16) branch_add_norm_kernel<<<n, row_threads(W), 0, s>>>(x, bs, (const __nv_bfloat16*)w, (const __nv_bfloat16*)b, w_offset, eps, W, (__nv_bfloat16*)h);
    else branch_add_norm_kernel<<<n, row_threads(W), 0, s>>>(x, bs, (const float*)w, (const float*)b, w_offset, eps, W, (float*)h);
    return launch_check(cudaGetLastError(), "branch_add_norm");
}

// ---- element-wise norms (tanh(alpha x) w + b): no row statistics, so everything between two sublayers is one pass over the row ----------
template <typename T>
__global__ void dyn_tanh_kernel(const float* __restrict__ x, int ldx, const T* __restrict__ w, const T* __restrict__ b, const T* __restrict__ alpha, int W,
                                float* __restrict__ y, T* __restrict__ y_t, const int32_t* __restrict__ rows) {
    const int i = blockIdx.x;
    const float* xr = x + (size_t)(rows ? rows[i] : i) * ldx;
    const float al = to_f(alpha[0]);
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < W; c += gridDim.y * blockDim.x) {
        const float v = fmaf(tanhf(al * xr[c]), to_f(w[c]), to_f(b[c]));
        if (y) y[(size_t)i * W + c] = v;
        if (y_t) y_t[(size_t)i * W + c] = from_f<T>(v);
    }
}

int launch_dyn_tanh(int dt, const float* x, int ldx, const DynNorm& nm, int n, int W, float* y, void* y_t, const int32_t* rows, cudaStream_t s) {
    if (n <= 0) return WF_OK;
    if (!nm.w || !nm.b || !nm.alpha) { set_error("dyn_tanh: weight, bias and alpha are needed"); return WF_ERR_INVALID; }
    const dim3 grid(n, n < 256 ? (W + 255) / 256 : 1);
    if (dt == WF_BF16) dyn_tanh_kernel<<<grid, 256, 0, s>>>(x, ldx, (const __nv_bfloat16*)nm.w, (const __nv_bfloat16*)nm.b, (const __nv_bfloat16*)nm.alpha, W, y, (__nv_bfloat16*)y_t, rows);
    else dyn_tanh_kernel<<<grid, 256, 0, s>>>(x, ldx, (const float*)nm.w, (const float*)nm.b, (const float*)nm.alpha, W, y, (float*)y_t, rows);
    return launch_check(cudaGetLastError(), "dyn_tanh");
}

template <typename T> __device__ __forceinline__ void load_n(const T* p, float (&v)[1]) { v[0] = to_f(p[0]); }
template <typename T> __device__ __forceinline__ void load_n(const T* p, float (&v)[4]) { const float4 q = load4(p); v[0] = q.x; v[1] = q.y; v[2] = q.z; v[3] = q.w; }
template <typename T> __device__ __forceinline__ void store_n(T* p, const float (&v)[1]) { p[0] = from_f<T>(v[0]); }
template <typename T> __device__ __forceinline__ void store_n(T* p, const float (&v)[4]) { store4(p, v); }

// v += / = tanh(alpha u) w + b for VEC channels at c
template <typename T, int VEC>
__device__ __forceinline__ void dyn_apply(const DynNorm& nm, int c, const float (&u)[VEC], float (&out)[VEC]) {
    float w[VEC], b[VEC];
    load_n((const T*)nm.w + c, w);
    load_n((const T*)nm.b + c, b);
    const float al = to_f(((const T*)nm.alpha)[0]);
#pragma unroll
    for (int e = 0; e < VEC; ++e) out[e] = fmaf(tanhf(al * u[e]), w[e], b[e]);
}

// grid (tokens, channel blocks).  VEC = 4: W a multiple of 4 (rows 16-byte aligned)
template <typename T, int VEC>
__global__ void __launch_bounds__(256) stream_step_kernel(float* __restrict__ x, StreamStep st, int W) {
    const int i = blockIdx.x, c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC;
    if (c >= W) return;
    const size_t at = (size_t)i * W + c;
    float v[VEC];
    if (st.init) {
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = 0.f;
    } else load_n(x + at, v);
    if (st.y || st.yexp) {
        float u[VEC], d[VEC];
        if (st.yexp) {
#pragma unroll
            for (int e = 0; e < VEC; ++e) u[e] = 0.f;
            for (int k = 0; k < st.top; ++k) {
                const size_t pi = (size_t)i * st.top + k;
                const float w = st.wts[pi];
                float q[VEC];
                load_n(st.yexp + (st.pair_row ? (size_t)st.pair_row[pi] : pi) * W + c, q);
#pragma unroll
                for (int e = 0; e < VEC; ++e) u[e] = fmaf(w, q[e], u[e]);
            }
            if (st.shared_y) {
                float q[VEC];
                load_n(st.shared_y + at, q);
#pragma unroll
                for (int e = 0; e < VEC; ++e) u[e] += q[e];
            }
        } else load_n(st.y + at, u);
        if (st.bias) {
            float q[VEC];
            load_n((const T*)st.bias + c, q);
#pragma unroll
            for (int e = 0; e < VEC; ++e) u[e] += q[e];
        }
        dyn_apply<T, VEC>(st.post, c, u, d);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] += d[e];
    }
    if (st.embed) {
        float q[VEC];
        load_n((const T*)st.embed + (size_t)st.tokens[i] * W + c, q);
#pragma unroll
        for (int e = 0; e < VEC; ++e) v[e] = fmaf(st.embed_scale, q[e], v[e]);
    }
    store_n(x + at, v);
    if (st.pre.w) {
        float h[VEC];
        dyn_apply<T, VEC>(st.pre, c, v, h);
        store_n((T*)st.h + at, h);
        if (st.hf) store_n(st.hf + at, h);
    }
}

int launch_stream_step(int dt, float* x, const StreamStep& st, int n, int W, cudaStream_t s) {
    if (n <= 0) return WF_OK;
    if (((st.y || st.yexp) && !st.post.w) || (st.y && st.yexp) || (st.yexp && (!st.wts || st.top < 1)) || (st.embed && !st.tokens) || (st.pre.w && !st.h)) {
        set_error("stream_step: inconsistent inputs"); return WF_ERR_INVALID;
    }
    const int vec = W % 4 == 0 ? 4 : 1, per = W / vec;
    const int threads = per >= 256 && n >= sm_count() ? 256 : (per > 64 ? 128 : 64);      // few tokens: more, smaller blocks
    const dim3 grid(n, (per + threads - 1) / threads);
    if (dt == WF_BF16) { if (vec == 4) stream_step_kernel<__nv_bfloat16, 4><<<grid, threads, 0, s>>>(x, st, W); else stream_step_kernel<__nv_bfloat16, 1><<<grid, threads, 0, s>>>(x, st, W); }
    else { if (vec == 4) stream_step_kernel<float, 4><<<grid, threads, 0, s>>>(x, st, W); else stream_step_kernel<float, 1><<<grid, threads, 0, s>>>(x, st, W); }
    return launch_check(cudaGetLastError(), "stream_step");
}

__global__ void softcap_kernel(float* __restrict__ z, size_t count, float cap) {
    for (size_t k = (size_t)blockIdx.x * blockDim.x + threadIdx.x; k < count; k += (size_t)gridDim.x * blockDim.x) z[k] = cap * tanhf(z[k] / cap);
}

int launch_softcap(float* z, size_t count, float cap, cudaStream_t s) {
    if (count == 0) return WF_OK;
    const int blocks = (int)((count + 255) / 256 > 4096 ? 4096 : (count + 255) / 256);
    softcap_kernel<<<blocks, 256, 0, s>>>(z, count, cap);
    return launch_check(cudaGetLastError(), "softcap");
}

// thread per (token, channel)
template <typename T>
__global__ void causal_taps_kernel(Batch b, const float* __restrict__ in, int ld_in, const T* __restrict__ w, int taps, int C,
                                   const float* __restrict__ state, size_t slot_stride, int identity, int silu, T* __restrict__ out_t, int ld_t,
                                   float* __restrict__ out_f, int ld_f, const T* __restrict__ bias) {
    const int i = blockIdx.x;
    const int sq = b.tok_seq[i];
    const int li = i - b.seq_start[sq];                    // index inside this step's portion
    const float* st = state + (size_t)b.seq_slot[sq] * slot_stride;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
        float acc = identity ? in[(size_t)i * ld_in + c] : 0.f;
        for (int j = 0; j < taps; ++j) {
            const int src = li - (taps - 1) + j;           // portion-relative index of the tap's input
            const float v = src >= 0 ? in[(size_t)(i - li + src) * ld_in + c] : st[(size_t)(src + taps - 1) * C + c];
            acc = fmaf(to_f(w[(size_t)c * taps + j]), v, acc);
        }
        if (bias) acc += to_f(bias[c]);
        if (silu) acc = silu_f(acc);
        if (out_t) out_t[(size_t)i * ld_t + c] = from_f<T>(acc);
        if (out_f) out_f[(size_t)i * ld_f + c] = acc;
    }
}

int launch_causal_taps(int dt, const Batch& b, const float* in, int ld_in, const void* w, int taps, int C, const float* state,
                       size_t slot_stride, int identity, int silu, void* out_t, int ld_t, float* out_f, int ld_f, cudaStream_t s, const void* bias) {
    if (b.n <= 0) return WF_OK;
    if (taps < 1) { set_error("causal_taps: taps %d", taps); return WF_ERR_INVALID; }
    dim3 grid(b.n, (C + 255) / 256 > 8 ? 8 : (C + 255) / 256);
    if (dt == WF_BF16) causal_taps_kernel<<<grid, 256, 0, s>>>(b, in, ld_in, (const __nv_bfloat16*)w, taps, C, state, slot_stride, identity, silu, (__nv_bfloat16*)out_t, ld_t, out_f, ld_f, (const __nv_bfloat16*)bias);
    else causal_taps_kernel<<<grid, 256, 0, s>>>(b, in, ld_in, (const float*)w, taps, C, state, slot_stride, identity, silu, (float*)out_t, ld_t, out_f, ld_f, (const float*)bias);
    return launch_check(cudaGetLastError(), "causal_taps");
}

// thread per (sequence, channel): state[k] <- input at portion index len - (taps - 1) + k, taken from the old state when that is negative.
// Ascending k is safe in place: entry k reads old entry len + k > k.
__global__ void taps_state_kernel(Batch b, const float* __restrict__ in, int ld_in, int taps, int C, float* __restrict__ state, size_t slot_stride,
                                  int skip_single) {
    const int sq = blockIdx.x;
    const int len = b.seq_len[sq], start = b.seq_start[sq];
    if (skip_single && len == 1) return;                 // rolled by the fused norm + taps kernel
    float* st = state + (size_t)b.seq_slot[sq] * slot_stride;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
        for (int k = 0; k < taps - 1; ++k) {
            const int src = len - (taps - 1) + k;
            st[(size_t)k * C + c] = src >= 0 ? in[(size_t)(start + src) * ld_in + c] : st[(size_t)(src + taps - 1) * C + c];
        }
    }
}

int launch_taps_state(const Batch& b, const float* in, int ld_in, int taps, int C, float* state, size_t slot_stride, cudaStream_t s, int skip_single) {
    if (b.nseq <= 0 || taps <= 1) return WF_OK;
    dim3 grid(b.nseq, (C + 255) / 256 > 8 ? 8 : (C + 255) / 256);
    taps_state_kernel<<<grid, 256, 0, s>>>(b, in, ld_in, taps, C, state, slot_stride, skip_single);
    return launch_check(cudaGetLastError(), "taps_state");
}

// ---- grouped RMS norm fused with the input convolution that follows it ---------------------------------------------------------
// One block per token: it normalises the token's own row and the taps - 1 rows before it (those inside this step's portion; earlier ones
// come normalised from the carried state), applies the taps, and writes the operand of the sublayer's matrix products.  Rows that the
// next step will need are also written as float (hn) for the state roll; a sequence that brings a single token rolls its state here.
constexpr int NTAPS_MAX = 8;

template <typename T>
__global__ void norm_taps_kernel(Batch b, const float* __restrict__ x, int ldx, const T* __restrict__ nw, int groups, float eps, const T* __restrict__ cw,
                                 int taps, int W, float* __restrict__ state, size_t slot_stride, T* __restrict__ out_t, int ld_t, float* __restrict__ hn) {
    __shared__ float red[NTAPS_MAX][33];
    __shared__ float inv[NTAPS_MAX * 32];            // [tap][group]
    const int i = blockIdx.x;
    const int sq = b.tok_seq[i];
    const int li = i - b.seq_start[sq], len = b.seq_len[sq];
    const int gw = W / groups;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw_ = blockDim.x >> 5;
    float* st = state + (size_t)b.seq_slot[sq] * slot_stride;
    for (int g = 0; g < groups; ++g) {
        float ss[NTAPS_MAX];
#pragma unroll
        for (int j = 0; j < NTAPS_MAX; ++j) ss[j] = 0.f;
        for (int c = threadIdx.x; c < gw; c += blockDim.x) {
#pragma unroll
            for (int j = 0; j < NTAPS_MAX; ++j) {
                const int src = li - (taps - 1) + j;
                if (j < taps && src >= 0) { const float v = x[(size_t)(i - li + src) * ldx + g * gw + c]; ss[j] += v * v; }
            }
        }
#pragma unroll
        for (int j = 0; j < NTAPS_MAX; ++j) {
            if (j < taps) { const float v = warp_sum(ss[j]); if (lane == 0) red[j][warp] = v; }
        }
        __syncthreads();
        if (threadIdx.x < taps) {
            float t = 0.f;
            for (int w = 0; w < nw_; ++w) t += red[threadIdx.x][w];
            inv[threadIdx.x * 32 + g] = 1.f / sqrtf(t / (float)gw + eps);
        }
        __syncthreads();
    }
    const bool keep = li >= len - (taps - 1);        // one of the last taps - 1 rows of the portion: the next step's state
    for (int c = threadIdx.x; c < W; c += blockDim.x) {
        const int g = c / gw;
        const float wn = to_f(nw[c]);
        float acc = 0.f, cur = 0.f, old[NTAPS_MAX];
#pragma unroll
        for (int j = 0; j < NTAPS_MAX; ++j) {
            if (j < taps) {
                const int src = li - (taps - 1) + j;
                float v;
                if (src >= 0) v = x[(size_t)(i - li + src) * ldx + c] * inv[j * 32 + g] * wn;
                else v = st[(size_t)(src + taps - 1) * W + c];
                old[j] = v;
                acc = fmaf(to_f(cw[(size_t)c * taps + j]), v, acc);
                if (j == taps - 1) cur = v;
            }
        }
        out_t[(size_t)i * ld_t + c] = from_f<T>(cur + acc);
        if (keep && hn) hn[(size_t)i * W + c] = cur;
        if (len == 1) {                               // old[j] is the input at distance taps - 1 - j: the new tail is old[1 .. taps - 1]
#pragma unroll
            for (int j = 1; j < NTAPS_MAX; ++j) if (j < taps) st[(size_t)(j - 1) * W + c] = old[j];
        }
    }
}

int launch_norm_taps(int dt, const Batch& b, const float* x, int ldx, const void* nw, int groups, float eps, const void* cw, int taps, int W, float* state,
                     size_t slot_stride, void* out_t, int ld_t, float* hn, cudaStream_t s) {
    if (b.n <= 0) return WF_OK;
    if (!norm_taps_usable(groups, taps, W)) { set_error("norm_taps: %d groups / %d taps are beyond the fused kernel", groups, taps); return WF_ERR_UNSUPPORTED; }
    const int threads = W >= 2048 ? 512 : (W >= 512 ? 256 : 128);
    if (dt == WF_BF16) norm_taps_kernel<<<b.n, threads, 0, s>>>(b, x, ldx, (const __nv_bfloat16*)nw, groups, eps, (const __nv_bfloat16*)cw, taps, W, state, slot_stride, (__nv_bfloat16*)out_t, ld_t, hn);
    else norm_taps_kernel<<<b.n, threads, 0, s>>>(b, x, ldx, (const float*)nw, groups, eps, (const float*)cw, taps, W, state, slot_stride, (float*)out_t, ld_t, hn);
    return launch_check(cudaGetLastError(), "norm_taps");
}

// ---- the same for many tokens: statistics once per row, then a fully parallel apply ------------------------------------------------
// inv[row][group] = 1 / sqrt(mean_group(x^2) + eps): one warp per (row, group)
__global__ void row_group_inv_rms_kernel(const float* __restrict__ x, int ldx, int n, int groups, int gw, float eps, float* __restrict__ inv) {
    const int wid = (blockIdx.x * blockDim.x + threadIdx.x) >> 5, lane = threadIdx.x & 31;
    if (wid >= n * groups) return;
    const int row = wid / groups, g = wid - row * groups;
    const float* p = x + (size_t)row * ldx + (size_t)g * gw;
    float ss = 0.f;
    for (int c = lane; c < gw; c += 32) { const float v = p[c]; ss += v * v; }
    ss = warp_sum(ss);
    if (lane == 0) inv[wid] = 1.f / sqrtf(ss / (float)gw + eps);
}

// thread per (token, 4 channels): the taps over rows normalised with the precomputed statistics (or taken from the carried state).
// VEC = 4 needs W, the group width and the row strides to be multiples of 4 (one group per thread, 16-byte loads); VEC = 1 takes anything.
template <typename T, int VEC>
__global__ void norm_taps_apply_kernel(Batch b, const float* __restrict__ x, int ldx, const float* __restrict__ inv, const T* __restrict__ nw, int groups,
                                       const T* __restrict__ cw, int taps, int W, const float* __restrict__ state, size_t slot_stride, T* __restrict__ out_t,
                                       int ld_t, float* __restrict__ hn) {
    const int i = blockIdx.x;
    const int sq = b.tok_seq[i];
    const int li = i - b.seq_start[sq], len = b.seq_len[sq];
    const int gw = W / groups;
    const float* st = state + (size_t)b.seq_slot[sq] * slot_stride;
    const bool keep = li >= len - (taps - 1);
    for (int c = (blockIdx.y * blockDim.x + threadIdx.x) * VEC; c < W; c += gridDim.y * blockDim.x * VEC) {
        const int g = c / gw;
        float wn[VEC], acc[VEC], cur[VEC];
#pragma unroll
        for (int v = 0; v < VEC; ++v) { wn[v] = to_f(nw[c + v]); acc[v] = 0.f; cur[v] = 0.f; }
        for (int j = 0; j < taps; ++j) {
            const int src = li - (taps - 1) + j;
            float val[VEC];
            if (src >= 0) {
                const float* xr = x + (size_t)(i - li + src) * ldx + c;
                const float iv = inv[(size_t)(i - li + src) * groups + g];
                if (VEC == 4) { const float4 q = *reinterpret_cast<const float4*>(xr); val[0] = q.x; val[1 % VEC] = q.y; val[2 % VEC] = q.z; val[3 % VEC] = q.w; }
                else val[0] = xr[0];
#pragma unroll
                for (int v = 0; v < VEC; ++v) val[v] *= iv * wn[v];
            } else {
                const float* sr = st + (size_t)(src + taps - 1) * W + c;
#pragma unroll
                for (int v = 0; v < VEC; ++v) val[v] = sr[v];
            }
#pragma unroll
            for (int v = 0; v < VEC; ++v) { acc[v] = fmaf(to_f(cw[(size_t)(c + v) * taps + j]), val[v], acc[v]); cur[v] = val[v]; }
        }
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
            out_t[(size_t)i * ld_t + c + v] = from_f<T>(cur[v] + acc[v]);
            if (keep && hn) hn[(size_t)i * W + c + v] = cur[v];
        }
    }
}

int launch_norm_taps_rows(int dt, const Batch& b, const float* x, int ldx, const void* nw, int groups, float eps, const void* cw, int taps, int W,
                          const float* state, size_t slot_stride, void* out_t, int ld_t, float* hn, float* inv, cudaStream_t s) {
    if (b.n <= 0) return WF_OK;
    if (groups < 1 || W % groups || taps < 1) { set_error("norm_taps_rows: %d groups / %d taps", groups, taps); return WF_ERR_INVALID; }
    const int warps = b.n * groups;
    row_group_inv_rms_kernel<<<(warps + 7) / 8, 256, 0, s>>>(x, ldx, b.n, groups, W / groups, eps, inv);
    if (int rc = launch_check(cudaGetLastError(), "row_group_inv_rms")) return rc;
    const bool vec = W % 4 == 0 && (W / groups) % 4 == 0 && ldx % 4 == 0 && (((uintptr_t)x) & 15) == 0;
    dim3 grid(b.n, vec ? (W + 1023) / 1024 : (W + 255) / 256);
    if (dt == WF_BF16) {
        if (vec) norm_taps_apply_kernel<__nv_bfloat16, 4><<<grid, 256, 0, s>>>(b, x, ldx, inv, (const __nv_bfloat16*)nw, groups, (const __nv_bfloat16*)cw, taps, W, state, slot_stride, (__nv_bfloat16*)out_t, ld_t, hn);
        else norm_taps_apply_kernel<__nv_bfloat16, 1><<<grid, 256, 0, s>>>(b, x, ldx, inv, (const __nv_bfloat16*)nw, groups, (const __nv_bfloat16*)cw, taps, W, state, slot_stride, (__nv_bfloat16*)out_t, ld_t, hn);
    } else {
        if (vec) norm_taps_apply_kernel<float, 4><<<grid, 256, 0, s>>>(b, x, ldx, inv, (const float*)nw, groups, (const float*)cw, taps, W, state, slot_stride, (float*)out_t, ld_t, hn);
        else norm_taps_apply_kernel<float, 1><<<grid, 256, 0, s>>>(b, x, ldx, inv, (const float*)nw, groups, (const float*)cw, taps, W, state, slot_stride, (float*)out_t, ld_t, hn);
    }
    return launch_check(cudaGetLastError(), "norm_taps_apply");
}

template <typename T>
__global__ void gate_mul_kernel(const float* __restrict__ x, int ldx, const float* __restrict__ g, int ldg, int act, int C, T* __restrict__ y, int ldy) {
    const int i = blockIdx.x;
    for (int c = blockIdx.y * blockDim.x + threadIdx.x; c < C; c += gridDim.y * blockDim.x) {
        const float z = g[(size_t)i * ldg + c];
        y[(size_t)i * ldy + c] = from_f<T>(x[(size_t)i * ldx + c] * (act == 2 ? 1.f : (act ? silu_f(z) : sigmoid_f(z))));
    }
}

int launch_gate_mul(int dt, const float* x, int ldx, const float* g, int ldg, int act, int n, int C, void* y, int ldy, cudaStream_t s) {
    if (n <= 0) return WF_OK;
    const dim3 grid(n, n < 64 ? (C + 255) / 256 : 1);
    if (dt == WF_BF16) gate_mul_kernel<<<grid, 256, 0, s>>>(x, ldx, g, ldg, act, C, (__nv_bfloat16*)y, ldy);
    else gate_mul_kernel<<<grid, 256, 0, s>>>(x, ldx, g, ldg, act, C, (float*)y, ldy);
    return launch_check(cudaGetLastError(), "gate_mul");
}

template <typename T>
__global__ void gather_rows_kernel(const T* __restrict__ src, int ld, const int32_t* __restrict__ rows, int W, T* __restrict__ dst) {
    const int i = blockIdx.x, r = rows[i];
    for (int c = threadIdx.x; c < W; c += blockDim.x) dst[(size_t)i * W + c] = r >= 0 ? src[(size_t)r * ld + c] : from_f<T>(0.f);
}

int launch_gather_rows(int dt, const void* src, int ld, const int32_t* rows, int P, int W, void* dst, cudaStream_t s) {
    if (P <= 0) return WF_OK;
    if (dt == WF_BF16) gather_rows_kernel<<<P, 256, 0, s>>>((const __nv_bfloat16*)src, ld, rows, W, (__nv_bfloat16*)dst);
    else gather_rows_kernel<<<P, 256, 0, s>>>((const float*)src, ld, rows, W, (float*)dst);
    return launch_check(cudaGetLastError(), "gather_rows");
}

template <typename T>
__global__ void transpose_heads_kernel(const T* __restrict__ in, int R, int C, T* __restrict__ out) {
    const size_t h = blockIdx.y;
    for (int idx = blockIdx.x * blockDim.x + threadIdx.x; idx < R * C; idx += gridDim.x * blockDim.x) {
        const int r = idx / C, c = idx % C;
        out[h * R * C + (size_t)c * R + r] = in[h * R * C + idx];
    }
}

int launch_transpose_heads(int dt, const void* in, int H, int R, int C, void* out, cudaStream_t s) {
    dim3 grid((R * C + 255) / 256 > 1024 ? 1024 : (R * C + 255) / 256, H);
    if (dt == WF_BF16) transpose_heads_kernel<<<grid, 256, 0, s>>>((const __nv_bfloat16*)in, R, C, (__nv_bfloat16*)out);
    else transpose_heads_kernel<<<grid, 256, 0, s>>>((const float*)in, R, C, (float*)out);
    return launch_check(cudaGetLastError(), "transpose_heads");
}

}  // namespace seq
}  // namespace wf
