// Parts that look the step's token ids up in tables of their own:
//
//   embedding with pairs of tokens      h[t,:] = scale * E[id_t,:] + P[row(id_(t-1), id_t),:]
//   input by token behind a product     out[t,j] = gelu_tanh(z[t,j]) * S[id_t, col0 + j]
//
// The token before an entry's first one is state of the request: one integer a slot.  The reference's embedding is a
// gather (crates/infer-worker/src/components/embed.rs:78-81); these stand beside it.
#include "common.cuh"

namespace {

template <typename T> __device__ __forceinline__ float4 load4(const T* p);
template <> __device__ __forceinline__ float4 load4<float>(const float* p) { return *reinterpret_cast<const float4*>(p); }
template <> __device__ __forceinline__ float4 load4<bf16>(const bf16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    const float2 a = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.x));
    const float2 b = __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(&u.y));
    return make_float4(a.x, a.y, b.x, b.y);
}

__device__ __forceinline__ int clamp_id(int id, int vocab) { return id < 0 ? 0 : (id >= vocab ? vocab - 1 : id); }

// A CTA a token.  The row of the pair (a, b) is (a * mul_prev + b * mul_cur) mod buckets in 64-bit; a token at position 0
// has row `buckets`, the table's last.  The token before an entry's first one comes from last_token[slot]; the CTA of an
// entry's first token is the only one that touches the slot: it reads it, then leaves the entry's last token there.
template <typename TE, typename TP, int V>
__global__ void embed_pairs_kernel(const int* __restrict__ ids, const int* __restrict__ positions, const int* __restrict__ cu_q,
                                   int entries, const int* __restrict__ slots, int* __restrict__ last_token,
                                   const TE* __restrict__ table, float scale, const TP* __restrict__ pairs,
                                   long long mul_prev, long long mul_cur, long long buckets, float* __restrict__ out, int tokens,
                                   int d, int vocab) {
    pdl_trigger();
    pdl_wait();
    const int t = blockIdx.x;
    __shared__ long long row_s;
    const int id = clamp_id(ids[t], vocab);
    if (threadIdx.x == 0) {
        int lo = t;                                            // the entry whose tokens t is among
        if (entries != tokens) {
            lo = 0;
            int hi = entries - 1;
            while (lo < hi) {
                const int mid = (lo + hi + 1) >> 1;
                if (cu_q[mid] <= t) lo = mid; else hi = mid - 1;
            }
        }
        int prev = t > 0 ? ids[t - 1] : 0;
        if (t == cu_q[lo]) {
            prev = last_token[slots[lo]];
            last_token[slots[lo]] = ids[cu_q[lo + 1] - 1];
        }
        row_s = positions[t] == 0 ? buckets : ((long long)clamp_id(prev, vocab) * mul_prev + (long long)id * mul_cur) % buckets;
    }
    __syncthreads();
    const TE* e = table + (size_t)id * d;
    const TP* p = pairs + (size_t)row_s * d;
    float* o = out + (size_t)t * d;
    for (int i = threadIdx.x * V; i < d; i += blockDim.x * V) {
        if (V == 4) {
            const float4 a = load4<TE>(e + i), b = load4<TP>(p + i);
            *reinterpret_cast<float4*>(o + i) = make_float4(fmaf(a.x, scale, b.x), fmaf(a.y, scale, b.y), fmaf(a.z, scale, b.z),
                                                            fmaf(a.w, scale, b.w));
        } else {
            o[i] = fmaf(to_f32<TE>(e[i]), scale, to_f32<TP>(p[i]));
        }
    }
}

__device__ __forceinline__ float gelu_tanh_f(float z) {
    return 0.5f * z * (1.0f + tanhf(0.7978845608028654f * (z + 0.044715f * z * z * z)));
}

template <typename TS, typename TO>
__global__ void token_gate_kernel(const float* __restrict__ z, int z_stride, const int* __restrict__ ids, const TS* __restrict__ table,
                                  int table_cols, int col0, int vocab, TO* __restrict__ out, int T, int n) {
    pdl_trigger();
    pdl_wait();
    const long long total = (long long)T * n;
    for (long long i = (long long)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += (long long)gridDim.x * blockDim.x) {
        const int t = (int)(i / n), j = (int)(i - (long long)t * n);
        const float e = to_f32<TS>(table[(size_t)clamp_id(ids[t], vocab) * table_cols + col0 + j]);
        out[i] = from_f32<TO>(gelu_tanh_f(z[(size_t)t * z_stride + j]) * e);
    }
}

}  // namespace

// table [vocab][d] and pairs [buckets + 1][d] of their dtypes, out fp32 [tokens][d]; cu_q [entries + 1], slots [entries],
// last_token [slots], positions and ids [tokens], all int32.
RI_API int ri_embed_pairs(const int* ids, const int* positions, const int* cu_q, int entries, const int* slots, int* last_token,
                          const void* table, int table_dtype, float scale, const void* pairs, int pairs_dtype, long long mul_prev,
                          long long mul_cur, long long buckets, float* out, int tokens, int d, int vocab, void* stream) {
    if (tokens <= 0) return 0;
    if (entries <= 0 || buckets <= 0 || mul_prev < 0 || mul_cur < 0) return (int)cudaErrorInvalidValue;
    cudaStream_t s = (cudaStream_t)stream;
    const auto at16 = [](const void* p) { return ((uintptr_t)p & 15) == 0; };
    const bool vec = d % 4 == 0 && at16(table) && at16(pairs) && at16(out);
#define RI_EP(TE, TP, V) RI_CHECKED(ri_launch(embed_pairs_kernel<TE, TP, V>, dim3(tokens), dim3(d / V >= 256 ? 256 : 128), 0, s, ids, \
        positions, cu_q, entries, slots, last_token, (const TE*)table, scale, (const TP*)pairs, mul_prev, mul_cur, buckets, out, \
        tokens, d, vocab))
#define RI_EP2(TE, TP) do { if (vec) RI_EP(TE, TP, 4); else RI_EP(TE, TP, 1); } while (0)
    if (table_dtype == RI_BF16) { if (pairs_dtype == RI_BF16) RI_EP2(bf16, bf16); else RI_EP2(bf16, float); }
    else { if (pairs_dtype == RI_BF16) RI_EP2(float, bf16); else RI_EP2(float, float); }
#undef RI_EP2
#undef RI_EP
    return ri_launch_status();
}

// z fp32 rows of z_stride, n columns; table [vocab][table_cols]; out [T][n].
RI_API int ri_token_gate(const float* z, int z_stride, const int* ids, const void* table, int table_dtype, int table_cols, int col0,
                         int vocab, void* out, int out_dtype, int T, int n, void* stream) {
    if (T <= 0) return 0;
    if (n <= 0 || col0 < 0 || col0 + n > table_cols) return (int)cudaErrorInvalidValue;
    cudaStream_t s = (cudaStream_t)stream;
    const long long nb = ((long long)T * n + 255) / 256, most = (long long)ri_device_sms() * 16;
    const dim3 grid((unsigned)(nb < most ? nb : most));
#define RI_TG(TS, TO) RI_CHECKED(ri_launch(token_gate_kernel<TS, TO>, grid, dim3(256), 0, s, z, z_stride, ids, (const TS*)table, \
        table_cols, col0, vocab, (TO*)out, T, n))
    if (table_dtype == RI_BF16) { if (out_dtype == RI_BF16) RI_TG(bf16, bf16); else RI_TG(bf16, float); }
    else { if (out_dtype == RI_BF16) RI_TG(float, bf16); else RI_TG(float, float); }
#undef RI_TG
    return ri_launch_status();
}
