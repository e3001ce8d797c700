// Parts of decoders that norm a sublayer's OUTPUT and nothing else (the sublayers read the residual stream itself), and
// of two of the mixers such blocks use:
//
//   norm of the output + residual add           h <- h + rms(y) * w;  act = round(h)
//     y a sublayer's output, or the weighted sum of a token's experts formed in the same launch
//   rotation of a projection's heads, in place  the first channels of every head turn by the position's angles
//   norm over parts of a row with a gate        out = rms_part(y) * w * silu(z), or rms_part(y * silu(z)) * w with
//                                               y = o (+ D_head * x)
//
// The stream, every norm, gate and rotation are fp32; what a matrix product reads is rounded once, at the end.  The
// reference engine has only the pre-norm block (crates/infer-worker/src/components/decoder_block.rs:13-32).
#include "common.cuh"

namespace {

template <typename T> __device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<bf16>(const bf16* p) {
    const uint2 v = *reinterpret_cast<const uint2*>(p);
    const float2 lo = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.x));
    const float2 hi = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&v.y));
    return make_float4(lo.x, lo.y, hi.x, hi.y);
}
template <typename T> __device__ __forceinline__ void store4(T* p, float4 v);
template <> __device__ __forceinline__ void store4<float>(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
template <> __device__ __forceinline__ void store4<bf16>(bf16* p, float4 v) {
    const __nv_bfloat162 lo = __floats2bfloat162_rn(v.x, v.y), hi = __floats2bfloat162_rn(v.z, v.w);
    uint2 u;
    u.x = *reinterpret_cast<const unsigned*>(&lo);
    u.y = *reinterpret_cast<const unsigned*>(&hi);
    *reinterpret_cast<uint2*>(p) = u;
}

// What a feed-forward of routed experts leaves for the kernel behind it: the experts' rows in expert order, where a
// token's rows lie, its weights, and a shared expert's row with a factor a token.
struct ExpertSum {
    const float* Y;              // [T * top][d]; null: the sublayer's output is given as it is
    const int* place;            // [T * top]
    const float* weights;        // [T * top]
    const float* shared;         // [T][d] or null
    const float* shared_gate;    // [T] or null (factor 1)
    int top;
    int* counts;                 // [E] put back to zero
    int E;
};

// One CTA a token; the row stays in shared memory between the sum of squares and the add (a thread reads back only
// what it wrote).  V = 4: four elements an access.
template <typename TD, typename TO, int V>
__global__ void norm_add_kernel(float* __restrict__ h, const TD* __restrict__ y, const float* __restrict__ w, int w_scalar,
                                float eps, TO* __restrict__ act, int d, ExpertSum es) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float row[];
    __shared__ float red[33];
    const size_t t = blockIdx.x;
    const int step = blockDim.x * V, first = threadIdx.x * V;
    float ss = 0.f;
    if (es.Y) {
        if (t == 0)
            for (int e = threadIdx.x; e < es.E; e += blockDim.x) es.counts[e] = 0;          // ready for the next step
        const float sg = es.shared_gate ? es.shared_gate[t] : 1.f;
        for (int i = first; i < d; i += step) {
            float a[V];
#pragma unroll
            for (int v = 0; v < V; ++v) a[v] = 0.f;
            for (int j = 0; j < es.top; ++j) {
                const float wj = es.weights[t * es.top + j];
                const float* src = es.Y + (size_t)es.place[t * es.top + j] * d + i;
                if (V == 4) {
                    const float4 x = load4<float>(src);
                    a[0] = fmaf(wj, x.x, a[0]); a[V > 1 ? 1 : 0] = fmaf(wj, x.y, a[V > 1 ? 1 : 0]);
                    a[V > 2 ? 2 : 0] = fmaf(wj, x.z, a[V > 2 ? 2 : 0]); a[V > 3 ? 3 : 0] = fmaf(wj, x.w, a[V > 3 ? 3 : 0]);
                } else {
                    a[0] = fmaf(wj, src[0], a[0]);
                }
            }
#pragma unroll
            for (int v = 0; v < V; ++v) {
                if (es.shared) a[v] = fmaf(sg, es.shared[t * d + i + v], a[v]);
                row[i + v] = a[v];
                ss += a[v] * a[v];
            }
        }
    } else {
        for (int i = first; i < d; i += step) {
            if (V == 4) {
                const float4 x = load4<TD>(y + t * d + i);
                *reinterpret_cast<float4*>(row + i) = x;
                ss += x.x * x.x + x.y * x.y + x.z * x.z + x.w * x.w;
            } else {
                const float x = to_f32<TD>(y[t * d + i]);
                row[i] = x;
                ss += x * x;
            }
        }
    }
    const float inv = 1.0f / sqrtf(block_sum(ss, red) / (float)d + eps);
    const float w0 = w_scalar ? w[0] : 0.f;
    for (int i = first; i < d; i += step) {
        if (V == 4) {
            const float4 x = *reinterpret_cast<float4*>(row + i), hv = load4<float>(h + t * d + i);
            const float4 g = w_scalar ? make_float4(w0, w0, w0, w0) : load4<float>(w + i);
            const float4 n = make_float4(hv.x + x.x * inv * g.x, hv.y + x.y * inv * g.y, hv.z + x.z * inv * g.z, hv.w + x.w * inv * g.w);
            store4<float>(h + t * d + i, n);
            if (act) store4<TO>(act + t * d + i, n);
        } else {
            const float n = h[t * d + i] + row[i] * inv * (w_scalar ? w0 : w[i]);
            h[t * d + i] = n;
            if (act) act[t * d + i] = from_f32<TO>(n);
        }
    }
}

// x [T][stride] fp32: `heads` heads of dk channels side by side; the first `rot` channels of each turn in place.
__global__ void rotate_cols_kernel(float* __restrict__ x, int stride, const int* __restrict__ positions,
                                   const float* __restrict__ cos_t, const float* __restrict__ sin_t, long long total,
                                   int heads, int dk, int rot, int interleaved) {
    pdl_trigger();
    pdl_wait();
    const int half = rot >> 1;
    for (long long e = (long long)blockIdx.x * blockDim.x + threadIdx.x; e < total; e += (long long)gridDim.x * blockDim.x) {
        const long long th = e / half;
        const int i = (int)(e - th * half);
        const long long t = th / heads;
        float* p = x + t * stride + (th - t * heads) * dk;
        const int ia = interleaved ? 2 * i : i, ib = interleaved ? 2 * i + 1 : i + half;
        const size_t at = (size_t)positions[t] * half + i;
        const float u = p[ia], v = p[ib], c = cos_t[at], s = sin_t[at];
        p[ia] = u * c - v * s;
        p[ib] = v * c + u * s;
    }
}

// A row of o [T][n_parts * n] in n_parts parts, each normed by its own root mean square.  With y = o (+ skip[channel / skip_group] * x):
//   gate_first:  g = y * silu(z);  out = g / rms(g) * w        else:  out = y / rms(y) * w * silu(z)
// (w null: 1; w has a number for every channel of the row).  GROUP threads a part, the part's values in shared memory.
template <typename TO, int GROUP>
__global__ void __launch_bounds__(256)
part_norm_gate_kernel(const float* __restrict__ o, const float* __restrict__ x, int x_stride, const float* __restrict__ skip,
                      int skip_group, const float* __restrict__ z, int z_stride, const float* __restrict__ w, float eps,
                      int gate_first, TO* __restrict__ out, long long items, int parts, int n) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) float sm[];
    __shared__ float red[33];
    constexpr int PER = 256 / GROUP;
    const int sub = threadIdx.x / GROUP, lane = threadIdx.x % GROUP;
    const long long item = (long long)blockIdx.x * PER + sub;
    if (GROUP == 32 && item >= items) return;                 // a whole warp (the block form has exactly one item a CTA)
    float* row = sm + (size_t)sub * n;
    const long long t = item / parts;
    const int c0 = (int)(item - t * parts) * n;
    const float* op = o + (size_t)t * parts * n + c0;
    const float* zp = z + (size_t)t * z_stride + c0;
    float ss = 0.f;
    for (int i = lane; i < n; i += GROUP) {
        float y = op[i];
        if (skip) y = fmaf(skip[(c0 + i) / skip_group], x[(size_t)t * x_stride + c0 + i], y);
        if (gate_first) {
            const float g = zp[i];
            y *= g / (1.0f + expf(-g));
        }
        row[i] = y;
        ss += y * y;
    }
    ss = GROUP == 32 ? warp_sum(ss) : block_sum(ss, red);
    const float inv = 1.0f / sqrtf(ss / (float)n + eps);
    TO* dst = out + (size_t)t * parts * n + c0;
    for (int i = lane; i < n; i += GROUP) {
        float y = row[i] * inv;
        if (w) y *= w[c0 + i];
        if (!gate_first) {
            const float g = zp[i];
            y *= g / (1.0f + expf(-g));
        }
        dst[i] = from_f32<TO>(y);
    }
}

}  // namespace

// h fp32 [rows][d] += rms(y) * w in place; act (may be null) gets the new h rounded to act_dtype.  w fp32: one number
// (w_scalar) or d of them.  y ([rows][d] of y_dtype) is given, or Y (fp32 [rows * top][d]) with place, weights and, each
// null or not, shared (fp32 [rows][d]) and shared_gate (fp32 [rows]): y = sum_j weights[j] Y[place[j]] + shared_gate * shared,
// and counts[0 .. E-1] are put back to zero.
RI_API int ri_norm_add(float* h, const void* y, int y_dtype, const float* w, int w_scalar, float eps, void* act, int act_dtype,
                       int rows, int d, const float* Y, const int* place, const float* weights, const float* shared,
                       const float* shared_gate, int top, int* counts, int E, void* stream) {
    if (rows <= 0) return 0;
    if ((y == nullptr) == (Y == nullptr) || (Y && (!place || !weights || !counts || top <= 0))) return (int)cudaErrorInvalidValue;
    cudaStream_t s = (cudaStream_t)stream;
    const size_t smem = (size_t)d * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    const ExpertSum es{Y, place, weights, shared, shared_gate, top, counts, E};
    auto at16 = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const bool vec = d % 4 == 0 && at16(h) && at16(y) && at16(act) && at16(Y) && at16(shared) && (w_scalar || at16(w));
    const int threads = d >= 2048 ? 512 : 256;
#define RI_NA(TD, TO, V) do { \
        static bool configured = false; \
        if (!configured && smem > 48 * 1024) { \
            cudaError_t e = cudaFuncSetAttribute(norm_add_kernel<TD, TO, V>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); \
            if (e != cudaSuccess) return (int)e; \
            configured = true; } \
        RI_CHECKED(ri_launch(norm_add_kernel<TD, TO, V>, dim3(rows), dim3(threads), smem, s, h, (const TD*)y, w, w_scalar, eps, \
            (TO*)act, d, es)); } while (0)
#define RI_NA2(TD, TO) do { if (vec) RI_NA(TD, TO, 4); else RI_NA(TD, TO, 1); } while (0)
    if (y_dtype == RI_BF16) { if (act_dtype == RI_BF16) RI_NA2(bf16, bf16); else RI_NA2(bf16, float); }
    else { if (act_dtype == RI_BF16) RI_NA2(float, bf16); else RI_NA2(float, float); }
#undef RI_NA2
#undef RI_NA
    return ri_launch_status();
}

RI_API int ri_rotate_cols(float* x, int stride, const int* positions, const float* cos_t, const float* sin_t, int tokens,
                          int heads, int dk, int rot, int interleaved, void* stream) {
    if (tokens <= 0 || rot <= 0) return 0;
    if (rot > dk || (rot & 1) || !cos_t || !sin_t) return (int)cudaErrorInvalidValue;
    const long long total = (long long)tokens * heads * (rot / 2), nb = (total + 255) / 256;
    const long long most = (long long)ri_device_sms() * 16;
    RI_CHECKED(ri_launch(rotate_cols_kernel, dim3((unsigned)(nb < most ? nb : most)), dim3(256), 0, (cudaStream_t)stream, x, stride,
                         positions, cos_t, sin_t, total, heads, dk, rot, interleaved));
    return ri_launch_status();
}

// o fp32 [rows][parts * n]; z fp32 rows of z_stride; w fp32 [parts * n] or null; skip fp32 [parts * n / skip_group] with
// x fp32 rows of x_stride, or null; out [rows][parts * n] of out_dtype.
RI_API int ri_part_norm_gate(const float* o, const float* x, int x_stride, const float* skip, int skip_group, const float* z,
                             int z_stride, const float* w, float eps, int gate_first, void* out, int out_dtype, int rows,
                             int parts, int n, void* stream) {
    if (rows <= 0) return 0;
    if (parts <= 0 || n <= 0 || (skip && (!x || skip_group <= 0)) || !z) return (int)cudaErrorInvalidValue;
    cudaStream_t s = (cudaStream_t)stream;
    const long long items = (long long)rows * parts;
    const bool warp = n <= 256;
    const size_t smem = (size_t)(warp ? 8 : 1) * n * sizeof(float);
    if (smem > 200 * 1024) return (int)cudaErrorInvalidValue;
    const dim3 grid((unsigned)(warp ? (items + 7) / 8 : items));
#define RI_PN(TO, G) do { \
        static bool configured = false; \
        if (!configured && smem > 48 * 1024) { \
            cudaError_t e = cudaFuncSetAttribute(part_norm_gate_kernel<TO, G>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024); \
            if (e != cudaSuccess) return (int)e; \
            configured = true; } \
        RI_CHECKED(ri_launch(part_norm_gate_kernel<TO, G>, grid, dim3(256), smem, s, o, x, x_stride, skip, skip_group, z, z_stride, w, \
            eps, gate_first, (TO*)out, items, parts, n)); } while (0)
    if (out_dtype == RI_BF16) { if (warp) RI_PN(bf16, 32); else RI_PN(bf16, 256); }
    else { if (warp) RI_PN(float, 32); else RI_PN(float, 256); }
#undef RI_PN
    return ri_launch_status();
}
