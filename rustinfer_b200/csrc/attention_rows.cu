// Paged attention on the tensor cores (mma.sync m16n8k16, bf16 operands, fp32 accumulate) for mixers whose keys
// and values differ in size or in number of heads, compiled for one RI_HEAD_DIM (size of a query and a key) and
// one RI_VALUE_DIM (size of a value), both multiples of 16.  It is the bfloat16 engine's kernel for prompt portions
// of the attention with several maps a head and of the attention over one cached row a token, and for single
// tokens of geometries the one-CTA-a-key-head kernel does not take.
//
// Scores are fp32 sums of exact products of bf16 q and k; scale, cap (cap * tanh(s / cap)), mask and the online
// softmax are fp32; the softmax weights enter the product with the values unrounded: a weight is cut into three
// bf16 pieces (8 + 8 + 8 bits of its significand, their sum is the weight) and every piece is multiplied with the
// bf16 values on the tensor cores with fp32 accumulation, the small pieces first.
//
// A CTA of four warps takes 64 rows of one key head, a row being (query token, query head of that key head), so
// the heads that share a key head share every tile that is loaded; a warp owns 16 rows.  Keys come in tiles of KT
// that start at multiples of KT from key 0 (the sums' order does not depend on how a prompt was cut), gathered page
// by page with cp.async into a double buffer.  Options as in the fp32-arithmetic kernel: `maps` attention maps a
// head (query heads [head][map], key heads [kv head][map], one set of values), values that are the keys' own first
// channels, a window, a term exp(sink_h) in the denominator, fp32 or bf16 output.  With `splits` > 1 the key tiles of
// every CTA are cut into that many ranges, a CTA each (grid z), which leave their unnormalised sums, maximum and sum
// in a scratch; a second kernel joins them.  That is for steps of few tiles over many keys (single tokens of a long
// context), where one CTA a tile would leave most SMs idle.  The reference has one
// attention kernel pair for one head size (crates/infer-backend-cuda/src/kernels/flash_attn_gqa/flash_attn_gqa.h:30).
#include "common.cuh"

#ifndef RI_HEAD_DIM
#error "compile with -DRI_HEAD_DIM=<key size> [-DRI_VALUE_DIM=<value size>]"
#endif
#ifndef RI_VALUE_DIM
#define RI_VALUE_DIM RI_HEAD_DIM
#endif

namespace {
constexpr int HD = RI_HEAD_DIM, VD = RI_VALUE_DIM;
static_assert(HD % 16 == 0 && HD >= 16 && HD <= 576, "key size: a multiple of 16, at most 576");
static_assert(VD % 16 == 0 && VD >= 16 && VD <= 256, "value size: a multiple of 16, at most 256");
constexpr int MT = 64;                         // rows a CTA
constexpr int THREADS = 128;
constexpr int KT = HD <= 128 ? 64 : 32;        // keys a tile
constexpr int KROW = HD + 8, VROW = VD + 8;    // padded rows: an odd count of 16-byte pieces, ldmatrix meets no conflict
constexpr int KCH = HD / 8, VCH = VD / 8;      // 16-byte pieces a row
constexpr int KS = HD / 16;                    // k-steps of q k^T
constexpr int NT = VD / 8;                     // n-tiles of the output
constexpr bool QREG = HD <= 128;               // the q fragments stay in registers
constexpr int PVG = 4;                         // value fragments (16 channels each) a group of the weights' products
constexpr float LOG2E = 1.4426950408889634f;

__device__ __forceinline__ void cp_async16(void* smem, const void* gmem, bool valid) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(smem);
    const int n = valid ? 16 : 0;              // 0 bytes read: the 16 bytes are filled with zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem), "r"(n));
}
// the same with the shared-memory address as the instructions take it
__device__ __forceinline__ unsigned smem_addr(const void* p) { return (unsigned)__cvta_generic_to_shared(p); }
__device__ __forceinline__ void cp_async16_at(unsigned s, const void* gmem) {
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16;\n" ::"r"(s), "l"(gmem));
}
__device__ __forceinline__ void cp_async16_at(unsigned s, const void* gmem, bool valid) {
    const int n = valid ? 16 : 0;
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;\n" ::"r"(s), "l"(gmem), "r"(n));
}
__device__ __forceinline__ void ldmatrix_x4_at(unsigned (&r)[4], unsigned s) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void ldmatrix_x4_trans_at(unsigned (&r)[4], unsigned s) {
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
// 2^x for x <= 0 or -inf on the special-function unit, one instruction
__device__ __forceinline__ float ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ void cp_async_commit() { asm volatile("cp.async.commit_group;\n" ::); }
template <int N> __device__ __forceinline__ void cp_async_wait() { asm volatile("cp.async.wait_group %0;\n" ::"n"(N)); }
__device__ __forceinline__ void ldmatrix_x4(unsigned (&r)[4], const void* p) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void ldmatrix_x4_trans(unsigned (&r)[4], const void* p) {
    const unsigned s = (unsigned)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];\n"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(s));
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const unsigned (&a)[4], unsigned b0, unsigned b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};\n"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ unsigned pack_bf16(float lo, float hi) {
    const __nv_bfloat162 v = __floats2bfloat162_rn(lo, hi);
    return *reinterpret_cast<const unsigned*>(&v);
}

struct Geometry {
    int Hq;                // query heads with their maps
    int Hkv;               // value heads
    int maps;              // maps a head
    int Gc;                // query heads of a key head a CTA takes
    int chunks;            // CTAs a key head's query heads are cut into
    int tpt;               // tokens a tile: MT / Gc
    int page_size;
    int window;            // 0: every earlier key
    int sink;              // the denominator holds exp(sink_values[h]) (null: exp(0)) besides the keys' terms
    int splits;            // ranges the key tiles of a CTA are cut into (grid z); > 1: results go through `part`
    int page_shift;        // log2 of page_size where that is a power of two, else -1
    float scale, softcap;  // softcap 0: scores are not capped
    const float* slopes;   // slopes[h] * (query position - key position) is taken off head h's scores (null: no such bias)
    const float* bias;     // bias[h * bias_len + min(query position - key position, bias_len - 1)] is added to head h's scores (null: none)
    int bias_len;
    int bias_span, bias_stride;    // bias in shared memory: distances it covers there, floats from one head to the next
    int block;             // > 0: a query sees only keys of its own block of that many positions (counted from 0)
    const float* gate;     // head h's output for token t times gate_scale * sigmoid(gate[t * gate_stride + h]) (null: as it is)
    int gate_stride;
    float gate_scale;
};
__device__ __forceinline__ float gate_of(const Geometry& gm, int t, int h) {
    return gm.gate ? gm.gate_scale / (1.0f + expf(-gm.gate[(size_t)t * gm.gate_stride + h])) : 1.f;
}

// keys k0 .. k0+KT-1 of key head `kh` (and, unless the values lie inside the keys, the values of value head `g`)
// into shared memory; keys outside [k_lo, k_hi) are zero-filled and their pages never looked up
template <bool VIK>
__device__ __forceinline__ void load_tile(bf16* Ks, bf16* Vs, const bf16* __restrict__ cache, const int* __restrict__ bt,
                                          int k0, int k_lo, int k_hi, size_t page_elems, size_t k_base, size_t v_base,
                                          int page_size, int page_shift) {
    constexpr int PIECES = KCH + (VIK ? 0 : VCH);
    for (int c = threadIdx.x; c < KT * PIECES; c += THREADS) {
        const int kk = c / PIECES, ch = c - kk * PIECES;
        const int key = k0 + kk;
        const bool ok = key >= k_lo && key < k_hi;
        const bf16* src = cache;
        if (ok) {
            const int blk = page_shift >= 0 ? key >> page_shift : key / page_size, off = key - blk * page_size;
            const bf16* page = cache + (size_t)bt[blk] * page_elems;
            src = ch < KCH ? page + k_base + (size_t)off * HD + ch * 8 : page + v_base + (size_t)off * VD + (ch - KCH) * 8;
        }
        bf16* dst = ch < KCH ? Ks + kk * KROW + ch * 8 : Vs + kk * VROW + (ch - KCH) * 8;
        cp_async16(dst, src, ok);
    }
}

// BIAS: the scores carry the learned distance bias (instantiations of their own: it costs registers).  1: the distances at
// which the bias still changes (and those a tile can meet beside them) lie in shared memory, a row a head, in units of log2,
// so that a score costs one load at a fixed offset and the multiply-add that scales it; 2: the table is read where it lies,
// the distance clamped to its end.  Tiles that lie wholly at the table's last entry or beyond take one number a row.
template <typename TO, bool VIK, int BIAS>
__global__ void __launch_bounds__(THREADS, VD <= 128 ? (VIK ? 4 : 3) : 1)      // values to 128 wide: three or four CTAs an SM
attention_rows_kernel(const bf16* __restrict__ q, int q_stride, TO* __restrict__ out, int out_stride,
                      const bf16* __restrict__ cache, const int* __restrict__ block_table, int table_stride,
                      const int* __restrict__ cu_q, const int* __restrict__ kv_len,
                      const int* __restrict__ tile_entry, const int* __restrict__ tile_tok0,
                      const float* __restrict__ sink_values, float* __restrict__ part, Geometry gm) {
    pdl_trigger();
    pdl_wait();
    extern __shared__ __align__(16) unsigned char smem_raw[];
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);            // [MT][KROW]
    bf16* KVs = Qs + MT * KROW;                              // [2 buffers][K: KT x KROW | V: KT x VROW]
    constexpr int BUF = KT * KROW + (VIK ? 0 : KT * VROW);

    const int b = tile_entry[blockIdx.x];
    if (b < 0) return;
    const int tok0 = tile_tok0[blockIdx.x];
    const int Hk = gm.Hkv * gm.maps;
    const int G = gm.Hq / Hk;                                // query heads a key head
    const int kh = blockIdx.y / gm.chunks, hc = blockIdx.y - kh * gm.chunks;
    const int kvh = kh / gm.maps, mp = kh - kvh * gm.maps;
    const int Gc = gm.Gc;
    const int g0 = hc * Gc, nheads = min(Gc, G - g0);        // heads g0 .. g0+nheads-1 of the key head's group
    const int q_begin = cu_q[b], q_len = cu_q[b + 1] - q_begin;
    const int pos0 = kv_len[b] - q_len;
    const int ntok = min(gm.tpt, q_len - tok0);
    if (ntok <= 0) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    // query head of the group's g-th head: ((kvh * G + g) * maps + mp)
    auto head_of = [&](int hh) { return (kvh * G + g0 + hh) * gm.maps + mp; };

    for (int c = tid; c < MT * KCH; c += THREADS) {
        const int r = c / KCH, ch = c - r * KCH;
        const int jj = r / Gc, hh = r - jj * Gc;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (jj < ntok && hh < nheads)
            v = *reinterpret_cast<const uint4*>(q + (size_t)(q_begin + tok0 + jj) * q_stride + (size_t)head_of(hh) * HD + ch * 8);
        *reinterpret_cast<uint4*>(Qs + r * KROW + ch * 8) = v;
    }

    const int p_first = pos0 + tok0, p_last = p_first + ntok - 1;
    int lo_tile = gm.window > 0 ? max(0, p_first - gm.window + 1) : 0;
    if (gm.block > 0) lo_tile = max(lo_tile, p_first / gm.block * gm.block);
    int t_begin = lo_tile / KT, t_end = p_last / KT + 1;
    if (gm.splits > 1) {
        // this CTA's range of the key tiles; it may be empty
        const int per = (t_end - t_begin + gm.splits - 1) / gm.splits;
        t_begin += blockIdx.z * per;
        t_end = min(t_end, t_begin + per);
    }
    const int* bt = block_table + (size_t)b * table_stride;
    const size_t page_elems = (size_t)gm.page_size * ((size_t)Hk * HD + (VIK ? 0 : (size_t)gm.Hkv * VD));
    const size_t k_base = (size_t)kh * gm.page_size * HD;
    const size_t v_base = (size_t)Hk * gm.page_size * HD + (size_t)kvh * gm.page_size * VD;

    if (t_begin < t_end)
        load_tile<VIK>(KVs, KVs + KT * KROW, cache, bt, t_begin * KT, lo_tile, p_last + 1, page_elems, k_base, v_base, gm.page_size, gm.page_shift);
    cp_async_commit();
    __syncthreads();                                          // Qs is written

    const int p_warp_first = p_first + (warp * 16) / Gc;     // position of the warp's first row
    float* Bs = reinterpret_cast<float*>(KVs + 2 * BUF);      // BIAS 1: [Gc][bias_stride]
    if (BIAS == 1) {
        const int need = min(gm.bias_span, max(p_last - lo_tile + 1, gm.bias_len));
        for (int hh = 0; hh < nheads; ++hh)
            for (int i = tid; i < need; i += THREADS)
                Bs[hh * gm.bias_stride + i] = gm.bias[(size_t)head_of(hh) * gm.bias_len + min(i, gm.bias_len - 1)] * LOG2E;
        // (read after the barrier that every tile has)
    }

    // this thread's two rows: 16 * warp + lane / 4 and that + 8
    int p_row[2], lo_row[2];
    bool ok_row[2];
    float m[2], l[2] = {0.f, 0.f}, slope[2] = {0.f, 0.f};
    int bias_row[2] = {0, 0};
#pragma unroll
    for (int i = 0; i < 2; ++i) {
        const int r = warp * 16 + (lane >> 2) + 8 * i;
        const int jj = r / Gc, hh = r - jj * Gc;
        ok_row[i] = jj < ntok && hh < nheads;
        if (gm.slopes && ok_row[i]) slope[i] = gm.slopes[head_of(hh)] * LOG2E;
        if (BIAS && ok_row[i]) bias_row[i] = BIAS == 1 ? hh * gm.bias_stride : head_of(hh) * gm.bias_len;
        p_row[i] = ok_row[i] ? p_first + jj : p_warp_first;
        lo_row[i] = gm.window > 0 ? max(0, p_row[i] - gm.window + 1) : 0;
        if (gm.block > 0) lo_row[i] = max(lo_row[i], p_row[i] / gm.block * gm.block);
        m[i] = -INFINITY;
        if (gm.sink && gm.splits == 1 && ok_row[i]) {           // with ranges, the join adds the term once
            // a term exp(sink_h) without a value: the maximum starts there and, in the one lane of four whose
            // partial sum stands for it, the sum at exp(sink_h - sink_h) = 1
            m[i] = (sink_values ? sink_values[head_of(hh)] : 0.f) * LOG2E;
            if ((lane & 3) == 0) l[i] = 1.f;
        }
    }
    // tiles between these two need no mask: the warp's first row sees their last key, its last row their first
    const int p_warp_last = p_first + min(ntok - 1, (warp * 16 + 15) / Gc);
    int lo_warp = gm.window > 0 ? max(0, p_warp_last - gm.window + 1) : 0;
    if (gm.block > 0) lo_warp = max(lo_warp, p_warp_last / gm.block * gm.block);
    const float scale2 = gm.scale * LOG2E;
    const bool warp_active = (warp * 16) / Gc < ntok;        // rows beyond the tile's tokens: nothing to do

    unsigned qf[QREG ? KS : 1][4];
    if (QREG) {
#pragma unroll
        for (int ks = 0; ks < (QREG ? KS : 1); ++ks)
            ldmatrix_x4(qf[ks], Qs + (warp * 16 + (lane & 15)) * KROW + ks * 16 + (lane >> 4) * 8);
    }
    float o[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;

    for (int t = t_begin; t < t_end; ++t) {
        const int buf = (t - t_begin) & 1;
        bf16* Ks = KVs + buf * BUF;
        bf16* Vs = VIK ? Ks : Ks + KT * KROW;
        constexpr int VSTRIDE = VIK ? KROW : VROW;
        if (t + 1 < t_end) {
            bf16* Kn = KVs + (buf ^ 1) * BUF;
            load_tile<VIK>(Kn, Kn + KT * KROW, cache, bt, (t + 1) * KT, lo_tile, p_last + 1, page_elems, k_base, v_base, gm.page_size, gm.page_shift);
            cp_async_commit();
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncthreads();
        if (warp_active) {
            float s[KT / 8][4];
#pragma unroll
            for (int n = 0; n < KT / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll
            for (int ks = 0; ks < KS; ++ks) {
                unsigned qk[4];
                if (!QREG) ldmatrix_x4(qk, Qs + (warp * 16 + (lane & 15)) * KROW + ks * 16 + (lane >> 4) * 8);
#pragma unroll
                for (int np = 0; np < KT / 16; ++np) {
                    unsigned kf[4];
                    ldmatrix_x4(kf, Ks + (np * 16 + (lane & 7) + (lane >> 4) * 8) * KROW + ks * 16 + ((lane >> 3) & 1) * 8);
                    mma_bf16(s[2 * np], QREG ? qf[QREG ? ks : 0] : qk, kf[0], kf[1]);
                    mma_bf16(s[2 * np + 1], QREG ? qf[QREG ? ks : 0] : qk, kf[2], kf[3]);
                }
            }
            // scale, cap, mask; everything from here on in units of log2
            const int key0 = t * KT + (lane & 3) * 2;
            float mx[2] = {-INFINITY, -INFINITY};
            if (t * KT + KT - 1 <= p_warp_first && t * KT >= lo_warp && !(gm.softcap > 0.f) && !gm.slopes) {
                if (BIAS && p_warp_first - (t * KT + KT - 1) >= gm.bias_len - 1) {
#pragma unroll
                    for (int i = 0; i < 2; ++i) {
                        const float far = BIAS == 1 ? Bs[bias_row[i] + gm.bias_len - 1] : __ldg(gm.bias + bias_row[i] + gm.bias_len - 1) * LOG2E;
#pragma unroll
                        for (int n = 0; n < KT / 8; ++n) {
#pragma unroll
                            for (int e = 0; e < 2; ++e) {
                                const float sc = fmaf(s[n][2 * i + e], scale2, far);
                                s[n][2 * i + e] = sc;
                                mx[i] = fmaxf(mx[i], sc);
                            }
                        }
                    }
                } else
#pragma unroll
                for (int i = 0; i < 2; ++i) {
                    const int d0 = p_row[i] - key0;           // distance of the thread's first key
                    const float* bp = BIAS == 1 ? Bs + bias_row[i] + d0 : nullptr;
#pragma unroll
                    for (int n = 0; n < KT / 8; ++n) {
#pragma unroll
                        for (int e = 0; e < 2; ++e) {
                            float sc = s[n][2 * i + e] * scale2;
                            if (BIAS == 1) sc = fmaf(s[n][2 * i + e], scale2, bp[-(n * 8 + e)]);
                            if (BIAS == 2)
                                sc = fmaf(s[n][2 * i + e], scale2, __ldg(gm.bias + bias_row[i] + min(d0 - n * 8 - e, gm.bias_len - 1)) * LOG2E);
                            s[n][2 * i + e] = sc;
                            mx[i] = fmaxf(mx[i], sc);
                        }
                    }
                }
            } else {
#pragma unroll
                for (int n = 0; n < KT / 8; ++n) {
#pragma unroll
                    for (int e = 0; e < 4; ++e) {
                        const int key = key0 + n * 8 + (e & 1);
                        const int i = e >> 1;
                        const bool seen = ok_row[i] && key <= p_row[i] && key >= lo_row[i];
                        float sc;
                        if (gm.softcap > 0.f) sc = gm.softcap * tanhf(s[n][e] * gm.scale / gm.softcap) * LOG2E;
                        else sc = s[n][e] * scale2;
                        sc -= slope[i] * (float)(p_row[i] - key);
                        if (BIAS == 1 && seen) sc = fmaf(s[n][e], scale2, Bs[bias_row[i] + min(p_row[i] - key, gm.bias_span - 1)]);
                        if (BIAS == 2 && seen)
                            sc = fmaf(s[n][e], scale2, __ldg(gm.bias + bias_row[i] + min(p_row[i] - key, gm.bias_len - 1)) * LOG2E);
                        s[n][e] = seen ? sc : -INFINITY;
                        mx[i] = fmaxf(mx[i], s[n][e]);
                    }
                }
            }
            float alpha[2], muse[2];
#pragma unroll
            for (int i = 0; i < 2; ++i) {
                mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 1));
                mx[i] = fmaxf(mx[i], __shfl_xor_sync(0xffffffffu, mx[i], 2));
                const float mnew = fmaxf(m[i], mx[i]);
                muse[i] = mnew == -INFINITY ? 0.f : mnew;
                alpha[i] = exp2f(m[i] - muse[i]);
                m[i] = mnew;
                l[i] *= alpha[i];
            }
#pragma unroll
            for (int n = 0; n < NT; ++n) {
                o[n][0] *= alpha[0]; o[n][1] *= alpha[0];
                o[n][2] *= alpha[1]; o[n][3] *= alpha[1];
            }
#pragma unroll
            for (int n = 0; n < KT / 8; ++n) {
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    s[n][e] = exp2f(s[n][e] - muse[e >> 1]);
                    l[e >> 1] += s[n][e];
                }
            }
#pragma unroll
            for (int kk = 0; kk < KT / 16; ++kk) {
                unsigned pa[3][4];
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    float a = s[2 * kk + (j >> 1)][(j & 1) * 2], c = s[2 * kk + (j >> 1)][(j & 1) * 2 + 1];
#pragma unroll
                    for (int piece = 0; piece < 3; ++piece) {
                        const unsigned packed = pack_bf16(a, c);
                        pa[piece][j] = packed;
                        a -= __uint_as_float(packed << 16);              // what the piece left out, exactly
                        c -= __uint_as_float(packed & 0xffff0000u);
                    }
                }
                // value fragments in groups of PVG: the products of one piece run over the whole group before the next
                // piece adds to the same accumulators, so consecutive products do not wait for one another
#pragma unroll
                for (int np0 = 0; np0 < NT / 2; np0 += PVG) {
                    unsigned vf[PVG][4];
#pragma unroll
                    for (int g = 0; g < PVG; ++g)
                        if (np0 + g < NT / 2)
                            ldmatrix_x4_trans(vf[g], Vs + (kk * 16 + (lane & 15)) * VSTRIDE + (np0 + g) * 16 + (lane >> 4) * 8);
#pragma unroll
                    for (int piece = 2; piece >= 0; --piece) {
#pragma unroll
                        for (int g = 0; g < PVG; ++g) {
                            if (np0 + g < NT / 2) {
                                mma_bf16(o[2 * (np0 + g)], pa[piece], vf[g][0], vf[g][1]);
                                mma_bf16(o[2 * (np0 + g) + 1], pa[piece], vf[g][2], vf[g][3]);
                            }
                        }
                    }
                }
            }
        }
        __syncthreads();                                      // all warps are done with this buffer
    }

#pragma unroll
    for (int i = 0; i < 2; ++i) {
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
        if (!ok_row[i]) continue;
        const int r = warp * 16 + (lane >> 2) + 8 * i;
        const int jj = r / Gc, hh = r - jj * Gc;
        if (gm.splits > 1) {
            float* dst = part + ((((size_t)blockIdx.x * gridDim.y + blockIdx.y) * MT + r) * gm.splits + blockIdx.z) * (VD + 2);
#pragma unroll
            for (int n = 0; n < NT; ++n)
                *reinterpret_cast<float2*>(dst + n * 8 + (lane & 3) * 2) = make_float2(o[n][2 * i], o[n][2 * i + 1]);
            if ((lane & 3) == 0) { dst[VD] = m[i]; dst[VD + 1] = l[i]; }
            continue;
        }
        const float inv = (l[i] > 0.f ? 1.f / l[i] : 0.f) * gate_of(gm, q_begin + tok0 + jj, head_of(hh));
        TO* dst = out + (size_t)(q_begin + tok0 + jj) * out_stride + (size_t)head_of(hh) * VD + (lane & 3) * 2;
#pragma unroll
        for (int n = 0; n < NT; ++n) {
            if constexpr (sizeof(TO) == 4) {
                *reinterpret_cast<float2*>(dst + n * 8) = make_float2(o[n][2 * i] * inv, o[n][2 * i + 1] * inv);
            } else {
                *reinterpret_cast<unsigned*>(dst + n * 8) = pack_bf16(o[n][2 * i] * inv, o[n][2 * i + 1] * inv);
            }
        }
    }
}

// Joins the ranges of one row of a tile, a warp a row: M = the largest maximum (the sink's exponent among them),
// L = sum l_z 2^(m_z - M) (+ 2^(sink - M)), out = sum acc_z 2^(m_z - M) / L; maxima are in units of log2.  Lane z
// holds range z's weight 2^(m_z - M) (ranges beyond 32 in a second turn); the sums run over the ranges in their order.
constexpr int MERGE_WARPS = 4;
template <typename TO>
__global__ void __launch_bounds__(MERGE_WARPS * 32)
attention_rows_merge_kernel(const float* __restrict__ part, TO* __restrict__ out, int out_stride,
                            const int* __restrict__ cu_q, const int* __restrict__ tile_entry,
                            const int* __restrict__ tile_tok0, const float* __restrict__ sink_values, Geometry gm) {
    pdl_trigger();
    pdl_wait();
    const int b = tile_entry[blockIdx.x];
    if (b < 0) return;
    const int tok0 = tile_tok0[blockIdx.x];
    const int Hk = gm.Hkv * gm.maps, G = gm.Hq / Hk, Gc = gm.Gc;
    const int kh = blockIdx.y / gm.chunks, hc = blockIdx.y - kh * gm.chunks;
    const int kvh = kh / gm.maps, mp = kh - kvh * gm.maps;
    const int g0 = hc * Gc, nheads = min(Gc, G - g0);
    const int q_begin = cu_q[b], ntok = min(gm.tpt, cu_q[b + 1] - q_begin - tok0);
    const int warp = threadIdx.x >> 5, lane = threadIdx.x & 31;
    const int r = blockIdx.z * MERGE_WARPS + warp;
    const int jj = r / Gc, hh = r - jj * Gc;
    if (r >= MT || jj >= ntok || hh >= nheads) return;
    const int head = (kvh * G + g0 + hh) * gm.maps + mp;
    constexpr int REC = VD + 2;
    const float* src = part + (((size_t)blockIdx.x * gridDim.y + blockIdx.y) * MT + r) * gm.splits * REC;
    const float sv = gm.sink ? (sink_values ? sink_values[head] : 0.f) * LOG2E : -INFINITY;
    // ranges lane and lane + 32 (splits <= 64)
    float mz[2], lz[2];
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        const int z = lane + 32 * k;
        mz[k] = z < gm.splits ? src[(size_t)z * REC + VD] : -INFINITY;
        lz[k] = z < gm.splits ? src[(size_t)z * REC + VD + 1] : 0.f;
    }
    float M = fmaxf(sv, fmaxf(mz[0], mz[1]));
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) M = fmaxf(M, __shfl_xor_sync(0xffffffffu, M, o));
    float wz[2], L = 0.f;
#pragma unroll
    for (int k = 0; k < 2; ++k) {
        wz[k] = mz[k] == -INFINITY ? 0.f : exp2f(mz[k] - M);
        L += lz[k] * wz[k];
    }
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) L += __shfl_xor_sync(0xffffffffu, L, o);
    if (gm.sink) L += exp2f(sv - M);
    const float inv = (L > 0.f ? 1.f / L : 0.f) * gate_of(gm, q_begin + tok0 + jj, head);
    TO* dst = out + (size_t)(q_begin + tok0 + jj) * out_stride + (size_t)head * VD;
    constexpr int DPL = (VD + 31) / 32;                       // channels a lane
    float acc[DPL];
#pragma unroll
    for (int i = 0; i < DPL; ++i) acc[i] = 0.f;
    for (int z = 0; z < gm.splits; ++z) {
        const float w = __shfl_sync(0xffffffffu, wz[z >> 5], z & 31);
        if (w == 0.f) continue;                               // an empty range: its sums were never written
#pragma unroll
        for (int i = 0; i < DPL; ++i) {
            const int d = lane + 32 * i;
            if (d < VD) acc[i] = fmaf(src[(size_t)z * REC + d], w, acc[i]);
        }
    }
#pragma unroll
    for (int i = 0; i < DPL; ++i) {
        const int d = lane + 32 * i;
        if (d >= VD) continue;
        if constexpr (sizeof(TO) == 4) dst[d] = acc[i] * inv; else dst[d] = __float2bfloat16(acc[i] * inv);
    }
}

// ------------------------------------------------------------------ entries of a single token
// A CTA takes up to 16 query heads of one key head of one entry (the rows of one m16 tile; the rest are zero rows), and its
// four warps take the key tiles in turn, each for itself: a warp has a double buffer of its own, fetches, multiplies and keeps
// a running maximum and sums of its own without meeting the others; their parts are joined once, at the end.  So all warps
// work however few heads share a key head, and a CTA has four tiles on their way at any time.  Arithmetic, options and
// `splits` as in the kernel above, whose join kernel serves this one too (row r of an entry is its head r of the key head's
// group, in chunks of 64).  LOW: no more than 8 rows, so the upper half of every fragment is skipped.
constexpr int KW = 16;                                        // keys a tile of a warp
template <bool VIK> constexpr size_t single_smem() {
    return ((size_t)16 * KROW + 4 * 2 * (size_t)KW * (KROW + (VIK ? 0 : VROW))) * sizeof(bf16);
}

template <typename TO, bool VIK, bool BIAS, bool LOW>
__global__ void __launch_bounds__(THREADS, VD <= 64 ? 5 : VD <= 128 ? (VIK ? 4 : 3) : 1)
attention_rows_single_kernel(const bf16* __restrict__ q, int q_stride, TO* __restrict__ out, int out_stride,
                             const bf16* __restrict__ cache, const int* __restrict__ block_table, int table_stride,
                             const int* __restrict__ cu_q, const int* __restrict__ kv_len, const int* __restrict__ entry_list,
                             const float* __restrict__ sink_values, float* __restrict__ part, Geometry gm) {
    pdl_trigger();
    pdl_wait();
    constexpr int BUF = KW * (KROW + (VIK ? 0 : VROW));
    constexpr int VSTRIDE = VIK ? KROW : VROW;
    constexpr int NI = LOW ? 1 : 2;                           // rows a thread keeps: lane / 4 and, unless LOW, that + 8
    extern __shared__ __align__(16) unsigned char smem_raw[];
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);             // [16][KROW]
    bf16* KVs = Qs + 16 * KROW;                               // [warp][2 buffers][K: KW x KROW | V: KW x VROW]
    __shared__ float ms[4][16], ls[4][16];

    const int b = entry_list[blockIdx.x];
    if (b < 0) return;
    const int t_q = cu_q[b];
    if (cu_q[b + 1] - t_q != 1) return;
    const int Hk = gm.Hkv * gm.maps, G = gm.Hq / Hk;
    const int chunks16 = (G + 15) / 16;
    const int kh = blockIdx.y / chunks16, g0 = (blockIdx.y - kh * chunks16) * 16;
    const int kvh = kh / gm.maps, mp = kh - kvh * gm.maps;
    const int nheads = min(16, G - g0);
    auto head_of = [&](int hh) { return (kvh * G + g0 + hh) * gm.maps + mp; };
    const int p = kv_len[b] - 1;
    int lo = gm.window > 0 ? max(0, p - gm.window + 1) : 0;
    if (gm.block > 0) lo = max(lo, p / gm.block * gm.block);
    int t_begin = lo / KW, t_end = p / KW + 1;
    if (gm.splits > 1) {                                      // this CTA's range of the key tiles; it may be empty
        const int per = (t_end - t_begin + gm.splits - 1) / gm.splits;
        t_begin += blockIdx.z * per;
        t_end = min(t_end, t_begin + per);
    }
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int* bt = block_table + (size_t)b * table_stride;
    const size_t page_elems = (size_t)gm.page_size * ((size_t)Hk * HD + (VIK ? 0 : (size_t)gm.Hkv * VD));
    const size_t k_base = (size_t)kh * gm.page_size * HD;
    const size_t v_base = (size_t)Hk * gm.page_size * HD + (size_t)kvh * gm.page_size * VD;
    bf16* mine = KVs + (size_t)warp * 2 * BUF;
    // a tile's 16 keys lie in one page, side by side, when pages are powers of two of 16 or more; else each is looked up
    const bool one_page = gm.page_shift >= 4;
    const unsigned mine_at = smem_addr(mine);
    // the page of the tile's keys (one page), or of key `lane % 16` of it; looked up a tile before the tile is fetched
    auto page_of = [&](int t) {
        if (t >= t_end) return 0;
        if (one_page) return bt[max(t * KW, lo) >> gm.page_shift];
        const int key = t * KW + (lane & (KW - 1));
        return key >= lo && key <= p ? bt[key / gm.page_size] : 0;
    };
    auto fetch = [&](int t, int pages, unsigned Kd) {
        const unsigned Vd = Kd + KW * KROW * (unsigned)sizeof(bf16);
        const int k0 = t * KW;
        if (one_page && k0 >= lo && k0 + KW - 1 <= p) {
            const bf16* page = cache + (size_t)pages * page_elems;
            const int off = k0 & (gm.page_size - 1);
            const bf16* kp = page + k_base + off * HD + lane * 8;
#pragma unroll
            for (int j = 0; j < KW * KCH / 32; ++j) {
                const int c = lane + 32 * j, kk = c / KCH, ch = c - kk * KCH;
                cp_async16_at(Kd + (kk * KROW + ch * 8) * (unsigned)sizeof(bf16), kp + 256 * j);
            }
            if (!VIK) {
                const bf16* vp = page + v_base + off * VD + lane * 8;
#pragma unroll
                for (int j = 0; j < KW * VCH / 32; ++j) {
                    const int c = lane + 32 * j, kk = c / VCH, ch = c - kk * VCH;
                    cp_async16_at(Vd + (kk * VROW + ch * 8) * (unsigned)sizeof(bf16), vp + 256 * j);
                }
            }
            return;
        }
        constexpr int PIECES = KCH + (VIK ? 0 : VCH);
#pragma unroll 1
        for (int c = lane; c < KW * PIECES; c += 32) {
            const int kk = c / PIECES, ch = c - kk * PIECES;
            const int key = k0 + kk;
            const bool ok = key >= lo && key <= p;
            const int other = __shfl_sync(0xffffffffu, pages, kk);
            const int pg = one_page ? pages : other;
            const int off = key % gm.page_size;
            const bf16* page = cache + (size_t)pg * page_elems;
            const bf16* src = VIK || ch < KCH ? page + k_base + off * HD + ch * 8 : page + v_base + off * VD + (ch - KCH) * 8;
            cp_async16_at((VIK || ch < KCH ? Kd + (kk * KROW + ch * 8) * (unsigned)sizeof(bf16)
                                           : Vd + (kk * VROW + (ch - KCH) * 8) * (unsigned)sizeof(bf16)), ok ? src : cache, ok);
        }
    };
    static_assert(KW * KCH % 32 == 0 && KW * VCH % 32 == 0, "every lane sends as many pieces");
    int t = t_begin + warp;
    int pages = page_of(t);
    if (t < t_end) fetch(t, pages, mine_at);
    cp_async_commit();
    pages = page_of(t + 4);
    for (int c = tid; c < 16 * KCH; c += THREADS) {
        const int r = c / KCH, ch = c - r * KCH;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (r < nheads) v = *reinterpret_cast<const uint4*>(q + (size_t)t_q * q_stride + (size_t)head_of(r) * HD + ch * 8);
        *reinterpret_cast<uint4*>(Qs + r * KROW + ch * 8) = v;
    }
    __syncthreads();
    unsigned qf[QREG ? KS : 1][4];
    if (QREG) {
#pragma unroll
        for (int ks = 0; ks < (QREG ? KS : 1); ++ks) ldmatrix_x4(qf[ks], Qs + (lane & 15) * KROW + ks * 16 + (lane >> 4) * 8);
    }
    float m[NI], l[NI], slope[NI], far[NI];
    const float* bias_row[NI];
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        const int hh = (lane >> 2) + 8 * i;
        const bool ok = hh < nheads;
        m[i] = -INFINITY;
        l[i] = 0.f;
        slope[i] = gm.slopes && ok ? gm.slopes[head_of(hh)] * LOG2E : 0.f;
        bias_row[i] = BIAS ? gm.bias + (size_t)head_of(ok ? hh : 0) * gm.bias_len : nullptr;
        far[i] = BIAS ? bias_row[i][gm.bias_len - 1] * LOG2E : 0.f;
    }
    float o[NT][4];
#pragma unroll
    for (int n = 0; n < NT; ++n) o[n][0] = o[n][1] = o[n][2] = o[n][3] = 0.f;
    const float scale2 = gm.scale * LOG2E;

    // where this lane's rows of the fragments lie in a buffer
    const unsigned k_lane = (((lane & 7) + (lane >> 4) * 8) * KROW + ((lane >> 3) & 1) * 8) * (unsigned)sizeof(bf16);
    const unsigned v_lane = (VIK ? 0u : KW * KROW * (unsigned)sizeof(bf16)) + ((lane & 15) * VSTRIDE + (lane >> 4) * 8) * (unsigned)sizeof(bf16);
    const unsigned q_lane = smem_addr(Qs) + ((lane & 15) * KROW + (lane >> 4) * 8) * (unsigned)sizeof(bf16);
    for (int it = 0; t < t_end; t += 4, ++it) {
        const unsigned kbuf = mine_at + (it & 1) * BUF * (unsigned)sizeof(bf16);
        const unsigned klane = kbuf + k_lane, vlane = kbuf + v_lane;
        if (t + 4 < t_end) {
            fetch(t + 4, pages, mine_at + ((it & 1) ^ 1) * BUF * (unsigned)sizeof(bf16));
            cp_async_commit();
            pages = page_of(t + 8);
            cp_async_wait<1>();
        } else {
            cp_async_wait<0>();
        }
        __syncwarp();
        float s[KW / 8][4];
#pragma unroll
        for (int n = 0; n < KW / 8; ++n) s[n][0] = s[n][1] = s[n][2] = s[n][3] = 0.f;
#pragma unroll
        for (int ks = 0; ks < KS; ++ks) {
            unsigned qk[4];
            if (!QREG) ldmatrix_x4_at(qk, q_lane + ks * 32);
#pragma unroll
            for (int np = 0; np < KW / 16; ++np) {
                unsigned kf[4];
                ldmatrix_x4_at(kf, klane + (np * 16 * KROW + ks * 16) * (unsigned)sizeof(bf16));
                mma_bf16(s[2 * np], QREG ? qf[QREG ? ks : 0] : qk, kf[0], kf[1]);
                mma_bf16(s[2 * np + 1], QREG ? qf[QREG ? ks : 0] : qk, kf[2], kf[3]);
            }
        }
        // scale, cap, bias, mask; everything from here on in units of log2
        const int key0 = t * KW + (lane & 3) * 2;
        const bool whole = t * KW >= lo && t * KW + KW - 1 <= p;
        const bool all_far = !BIAS || p - (t * KW + KW - 1) >= gm.bias_len - 1;
        float alpha[NI];
        bool grown = false;
        if (whole && all_far && !(gm.softcap > 0.f) && !gm.slopes) {
#pragma unroll
            for (int i = 0; i < NI; ++i) {
#pragma unroll
                for (int n = 0; n < KW / 8; ++n) {
                    s[n][2 * i] = fmaf(s[n][2 * i], scale2, far[i]);
                    s[n][2 * i + 1] = fmaf(s[n][2 * i + 1], scale2, far[i]);
                }
            }
        } else {
#pragma unroll
            for (int i = 0; i < NI; ++i) {
#pragma unroll
                for (int n = 0; n < KW / 8; ++n) {
#pragma unroll
                    for (int e = 0; e < 2; ++e) {
                        const int key = key0 + n * 8 + e;
                        const bool seen = key >= lo && key <= p;
                        float sc = s[n][2 * i + e];
                        if (gm.softcap > 0.f) sc = gm.softcap * tanhf(sc * gm.scale / gm.softcap) * LOG2E;
                        else sc *= scale2;
                        if (gm.slopes) sc -= slope[i] * (float)(p - key);
                        if (BIAS && seen) sc += __ldg(bias_row[i] + min(p - key, gm.bias_len - 1)) * LOG2E;
                        s[n][2 * i + e] = seen ? sc : -INFINITY;
                    }
                }
            }
        }
#pragma unroll
        for (int i = 0; i < NI; ++i) {
            float mx = -INFINITY;
#pragma unroll
            for (int n = 0; n < KW / 8; ++n) mx = fmaxf(mx, fmaxf(s[n][2 * i], s[n][2 * i + 1]));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 1));
            mx = fmaxf(mx, __shfl_xor_sync(0xffffffffu, mx, 2));
            grown |= mx > m[i];
            const float mnew = fmaxf(m[i], mx);               // a tile holds a seen key at least: it is finite
            alpha[i] = ex2(m[i] - mnew);
            m[i] = mnew;
            l[i] *= alpha[i];
#pragma unroll
            for (int n = 0; n < KW / 8; ++n) {
#pragma unroll
                for (int e = 0; e < 2; ++e) {
                    s[n][2 * i + e] = ex2(s[n][2 * i + e] - mnew);
                    l[i] += s[n][2 * i + e];
                }
            }
        }
        if (__any_sync(0xffffffffu, grown)) {                 // some row's maximum has grown
#pragma unroll
            for (int i = 0; i < NI; ++i) {
#pragma unroll
                for (int n = 0; n < NT; ++n) { o[n][2 * i] *= alpha[i]; o[n][2 * i + 1] *= alpha[i]; }
            }
        }
#pragma unroll
        for (int kk = 0; kk < KW / 16; ++kk) {
            unsigned pa[3][4];
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                if (LOW && (j & 1)) {
                    pa[0][j] = pa[1][j] = pa[2][j] = 0u;
                    continue;
                }
                float a = s[2 * kk + (j >> 1)][(j & 1) * 2], c = s[2 * kk + (j >> 1)][(j & 1) * 2 + 1];
#pragma unroll
                for (int piece = 0; piece < 3; ++piece) {
                    const unsigned packed = pack_bf16(a, c);
                    pa[piece][j] = packed;
                    a -= __uint_as_float(packed << 16);
                    c -= __uint_as_float(packed & 0xffff0000u);
                }
            }
#pragma unroll
            for (int np0 = 0; np0 < NT / 2; np0 += PVG) {
                unsigned vf[PVG][4];
#pragma unroll
                for (int g = 0; g < PVG; ++g)
                    if (np0 + g < NT / 2)
                        ldmatrix_x4_trans_at(vf[g], vlane + (kk * 16 * VSTRIDE + (np0 + g) * 16) * (unsigned)sizeof(bf16));
#pragma unroll
                for (int piece = 2; piece >= 0; --piece) {
#pragma unroll
                    for (int g = 0; g < PVG; ++g) {
                        if (np0 + g < NT / 2) {
                            mma_bf16(o[2 * (np0 + g)], pa[piece], vf[g][0], vf[g][1]);
                            mma_bf16(o[2 * (np0 + g) + 1], pa[piece], vf[g][2], vf[g][3]);
                        }
                    }
                }
            }
        }
        __syncwarp();                                         // the buffer is free for the tile after the next
    }
    // the warps' parts meet in shared memory (a warp's rows lie in its own buffers), joined in the warps' order
    float* po = reinterpret_cast<float*>(mine);               // [16][VD]
#pragma unroll
    for (int i = 0; i < NI; ++i) {
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 1);
        l[i] += __shfl_xor_sync(0xffffffffu, l[i], 2);
        const int r = (lane >> 2) + 8 * i;
        if ((lane & 3) == 0) { ms[warp][r] = m[i]; ls[warp][r] = l[i]; }
#pragma unroll
        for (int n = 0; n < NT; ++n)
            *reinterpret_cast<float2*>(po + r * VD + n * 8 + (lane & 3) * 2) = make_float2(o[n][2 * i], o[n][2 * i + 1]);
    }
    __syncthreads();
    const int chunk = g0 / gm.Gc, row0 = g0 - chunk * gm.Gc;  // where the rows lie in the records the join kernel reads
    for (int e = tid; e < nheads * VD; e += THREADS) {
        const int r = e / VD, d = e - r * VD;
        const bool sink = gm.sink && gm.splits == 1;          // with ranges, the join adds the term once
        const float sv = sink ? (sink_values ? sink_values[head_of(r)] : 0.f) * LOG2E : -INFINITY;
        const float M = fmaxf(sv, fmaxf(fmaxf(ms[0][r], ms[1][r]), fmaxf(ms[2][r], ms[3][r])));
        float acc = 0.f, L = sink ? exp2f(sv - M) : 0.f;
#pragma unroll
        for (int w = 0; w < 4; ++w) {
            const float wt = ms[w][r] == -INFINITY ? 0.f : exp2f(ms[w][r] - M);
            L = fmaf(ls[w][r], wt, L);
            acc = fmaf(reinterpret_cast<const float*>(KVs + (size_t)w * 2 * BUF)[r * VD + d], wt, acc);
        }
        if (gm.splits > 1) {
            float* dst = part + ((((size_t)blockIdx.x * (Hk * gm.chunks) + kh * gm.chunks + chunk) * MT + row0 + r) * gm.splits
                                 + blockIdx.z) * (VD + 2);
            dst[d] = acc;
            if (d == 0) { dst[VD] = M; dst[VD + 1] = L; }
        } else {
            out[(size_t)t_q * out_stride + (size_t)head_of(r) * VD + d] =
                from_f32<TO>((L > 0.f ? acc / L : 0.f) * gate_of(gm, t_q, head_of(r)));
        }
    }
}

constexpr size_t BIAS_SMEM = 24 * 1024;        // most shared memory the bias takes
template <typename TO, bool VIK, int BIAS>
int launch(const void* q, int q_stride, void* out, int out_stride, const void* cache, const int* block_table,
           int table_stride, const int* cu_q, const int* kv_len, const int* tile_entry, const int* tile_tok0,
           int n_tiles, const float* sink_values, float* part, const Geometry& gm, cudaStream_t s) {
    static bool configured = false;
    constexpr size_t base = ((size_t)MT * KROW + 2 * ((size_t)KT * KROW + (VIK ? 0 : (size_t)KT * VROW))) * sizeof(bf16);
    const size_t smem = base + (BIAS == 1 ? (size_t)gm.Gc * gm.bias_stride * sizeof(float) : 0);
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(attention_rows_kernel<TO, VIK, BIAS>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             (int)(base + (BIAS == 1 ? BIAS_SMEM : 0)));
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    dim3 grid(n_tiles, gm.Hkv * gm.maps * gm.chunks, gm.splits);
    RI_CHECKED(ri_launch(attention_rows_kernel<TO, VIK, BIAS>, grid, dim3(THREADS), smem, s, (const bf16*)q, q_stride, (TO*)out,
                         out_stride, (const bf16*)cache, block_table, table_stride, cu_q, kv_len, tile_entry, tile_tok0,
                         sink_values, part, gm));
    if (gm.splits > 1)
        RI_CHECKED(ri_launch(attention_rows_merge_kernel<TO>, dim3(grid.x, grid.y, MT / MERGE_WARPS), dim3(MERGE_WARPS * 32), 0, s,
                             (const float*)part, (TO*)out, out_stride, cu_q, tile_entry, tile_tok0, sink_values, gm));
    return ri_launch_status();
}

template <typename TO, bool VIK, bool BIAS, bool LOW>
int launch_single(const void* q, int q_stride, void* out, int out_stride, const void* cache, const int* block_table,
                  int table_stride, const int* cu_q, const int* kv_len, const int* entry_list, const int* zeros, int n_entries,
                  const float* sink_values, float* part, const Geometry& gm, cudaStream_t s) {
    static bool configured = false;
    constexpr size_t smem = single_smem<VIK>();
    static_assert(smem <= 220 * 1024, "the warps' buffers fit an SM");
    if (!configured) {
        cudaError_t e = cudaFuncSetAttribute(attention_rows_single_kernel<TO, VIK, BIAS, LOW>, cudaFuncAttributeMaxDynamicSharedMemorySize,
                                             (int)smem);
        if (e != cudaSuccess) return (int)e;
        configured = true;
    }
    const int Hk = gm.Hkv * gm.maps, G = gm.Hq / Hk;
    dim3 grid(n_entries, Hk * ((G + 15) / 16), gm.splits);
    RI_CHECKED(ri_launch(attention_rows_single_kernel<TO, VIK, BIAS, LOW>, grid, dim3(THREADS), smem, s, (const bf16*)q, q_stride, (TO*)out,
                         out_stride, (const bf16*)cache, block_table, table_stride, cu_q, kv_len, entry_list, sink_values, part, gm));
    if (gm.splits > 1)
        RI_CHECKED(ri_launch(attention_rows_merge_kernel<TO>, dim3(n_entries, Hk * gm.chunks, (gm.Gc + MERGE_WARPS - 1) / MERGE_WARPS),
                             dim3(MERGE_WARPS * 32), 0, s, (const float*)part, (TO*)out, out_stride, cu_q, entry_list, zeros, sink_values, gm));
    return ri_launch_status();
}
}  // namespace

RI_API int ri_attention_rows_head_dim() { return HD; }
RI_API int ri_attention_rows_value_dim() { return VD; }

// Query heads of a key head one CTA takes: all of them up to 64 (then MT / that many tokens a tile), else 64.
RI_API int ri_attention_rows_heads_per_cta(int Hq, int Hkv, int maps) {
    if (Hkv <= 0 || maps <= 0 || Hq % (Hkv * maps)) return 0;
    const int G = Hq / (Hkv * maps);
    return G < MT ? G : MT;
}

// Tokens of one tile: tile_tok0 counts in these.
RI_API int ri_attention_rows_tokens_per_tile(int Hq, int Hkv, int maps) {
    const int gc = ri_attention_rows_heads_per_cta(Hq, Hkv, maps);
    return gc > 0 ? MT / gc : 0;
}

// CTAs of the attention kernel that fit an SM at once (0: the question failed), for the choice of the key ranges.
RI_API int ri_attention_rows_ctas_per_sm(int value_in_key, int out_f32) {
    int n = 0;
    cudaError_t e = cudaErrorInvalidValue;
#define RI_ROWS_OCC(TO, VIK) do { \
        const size_t smem = ((size_t)MT * KROW + 2 * ((size_t)KT * KROW + (VIK ? 0 : (size_t)KT * VROW))) * sizeof(bf16); \
        e = cudaFuncSetAttribute(attention_rows_kernel<TO, VIK, 0>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        if (e == cudaSuccess) e = cudaOccupancyMaxActiveBlocksPerMultiprocessor(&n, attention_rows_kernel<TO, VIK, 0>, THREADS, smem); \
    } while (0)
    if (value_in_key) {
        if constexpr (VD <= HD) { if (out_f32) RI_ROWS_OCC(float, true); else RI_ROWS_OCC(bf16, true); }
    } else {
        if (out_f32) RI_ROWS_OCC(float, false); else RI_ROWS_OCC(bf16, false);
    }
#undef RI_ROWS_OCC
    return e == cudaSuccess ? n : 0;
}

// q [T][q_stride] bf16, head h at column h*HD; out rows of out_stride, head h at column h*VD, fp32 (out_f32) or bf16.
// cache: per page the keys [key head][slot][HD], then (unless value_in_key) the values [value head][slot][VD], bf16,
// every page starting on a 16-byte boundary.  tile_entry[i]: batch entry of tile i (-1: skip), tile_tok0[i] its first
// token within the entry; a tile holds ri_attention_rows_tokens_per_tile tokens.  splits > 1: the key tiles of every CTA
// in that many ranges through `part`, fp32 [n_tiles][key heads * chunks][64 rows][splits][VD + 2], and a second launch.
RI_API int ri_attention_rows(const void* q, int q_stride, void* out, int out_stride, const void* cache,
                             const int* block_table, int table_stride, const int* cu_q, const int* kv_len,
                             const int* tile_entry, const int* tile_tok0, int n_tiles, int Hq, int Hkv, int page_size,
                             float scale, int window, int sink, float softcap, const float* sink_values, int maps,
                             int value_in_key, int out_f32, int splits, float* part, const float* slopes,
                             const float* bias, int bias_len, int block, const float* gate, int gate_stride, float gate_scale,
                             void* stream) {
    if (n_tiles <= 0) return 0;
    if (bias && bias_len <= 0) return (int)cudaErrorInvalidValue;
    if (splits < 1 || splits > 64 || (splits > 1 && !part)) return (int)cudaErrorInvalidValue;
    const int gc = ri_attention_rows_heads_per_cta(Hq, Hkv, maps);
    if (gc <= 0 || (value_in_key && (maps != 1 || VD > HD)) || q_stride % 8) return (int)cudaErrorInvalidValue;
    const int G = Hq / (Hkv * maps);
    Geometry gm{Hq, Hkv, maps, gc, (G + gc - 1) / gc, MT / gc, page_size, window, sink, splits, -1, scale, softcap, slopes,
                bias, bias_len, 0, 0, block, gate, gate_stride, gate_scale};
    for (int sh = 0; sh < 20; ++sh)
        if (page_size == 1 << sh) gm.page_shift = sh;
    // distances the bias must be at hand for: those before the table's last entry and, from there on, what a tile that
    // starts before it can still meet; fewer where the block or the window ends earlier
    if (bias && bias_len < (1 << 20)) {
        int span = bias_len + KT + MT;
        if (block > 0 && block < span) span = block;
        if (window > 0 && window < span) span = window;
        const int stride = (span + 31) / 32 * 32 + 8;         // heads 8 banks apart: the lanes of a warp read without conflict
        if ((size_t)gc * stride * sizeof(float) <= BIAS_SMEM) { gm.bias_span = span; gm.bias_stride = stride; }
    }
    cudaStream_t s = (cudaStream_t)stream;
    if (bias && value_in_key) return (int)cudaErrorNotSupported;
    if (bias && (softcap > 0.f || slopes)) return (int)cudaErrorNotSupported;
#define RI_ROWS_GO(TO, VIK, BIAS) launch<TO, VIK, BIAS>(q, q_stride, out, out_stride, cache, block_table, table_stride, cu_q, kv_len, \
                                            tile_entry, tile_tok0, n_tiles, sink_values, part, gm, s)
    if (value_in_key) {
        if constexpr (VD <= HD) return out_f32 ? RI_ROWS_GO(float, true, 0) : RI_ROWS_GO(bf16, true, 0);
        return (int)cudaErrorInvalidValue;
    }
    if (bias && gm.bias_span) return out_f32 ? RI_ROWS_GO(float, false, 1) : RI_ROWS_GO(bf16, false, 1);
    if (bias) return out_f32 ? RI_ROWS_GO(float, false, 2) : RI_ROWS_GO(bf16, false, 2);
    return out_f32 ? RI_ROWS_GO(float, false, 0) : RI_ROWS_GO(bf16, false, 0);
#undef RI_ROWS_GO
}

// CTAs of the kernel for single tokens that fit an SM at once (0: the question failed).
RI_API int ri_attention_rows_single_ctas_per_sm(int value_in_key, int out_f32) {
    int n = 0;
    cudaError_t e = cudaErrorInvalidValue;
#define RI_SINGLE_OCC(TO, VIK) do { \
        constexpr size_t smem = single_smem<VIK>(); \
        e = cudaFuncSetAttribute(attention_rows_single_kernel<TO, VIK, false, false>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem); \
        if (e == cudaSuccess) e = cudaOccupancyMaxActiveBlocksPerMultiprocessor(&n, attention_rows_single_kernel<TO, VIK, false, false>, \
                                                                                THREADS, smem); \
    } while (0)
    if (value_in_key) {
        if constexpr (VD <= HD) { if (out_f32) RI_SINGLE_OCC(float, true); else RI_SINGLE_OCC(bf16, true); }
    } else {
        if (out_f32) RI_SINGLE_OCC(float, false); else RI_SINGLE_OCC(bf16, false);
    }
#undef RI_SINGLE_OCC
    return e == cudaSuccess ? n : 0;
}

// Entries that bring a single token (entry_list[i], -1: skip; zeros: as many zeros, for the join kernel).  Arguments as
// ri_attention_rows; `part` has its layout with n_entries for n_tiles.
RI_API int ri_attention_rows_single(const void* q, int q_stride, void* out, int out_stride, const void* cache,
                                    const int* block_table, int table_stride, const int* cu_q, const int* kv_len,
                                    const int* entry_list, const int* zeros, int n_entries, int Hq, int Hkv, int page_size,
                                    float scale, int window, int sink, float softcap, const float* sink_values, int maps,
                                    int value_in_key, int out_f32, int splits, float* part, const float* slopes,
                                    const float* bias, int bias_len, int block, const float* gate, int gate_stride, float gate_scale,
                                    void* stream) {
    if (n_entries <= 0) return 0;
    if (bias && bias_len <= 0) return (int)cudaErrorInvalidValue;
    if (splits < 1 || splits > 64 || (splits > 1 && (!part || !zeros))) return (int)cudaErrorInvalidValue;
    const int gc = ri_attention_rows_heads_per_cta(Hq, Hkv, maps);
    if (gc <= 0 || (value_in_key && (maps != 1 || VD > HD)) || q_stride % 8) return (int)cudaErrorInvalidValue;
    if (bias && value_in_key) return (int)cudaErrorNotSupported;
    const int G = Hq / (Hkv * maps);
    Geometry gm{Hq, Hkv, maps, gc, (G + gc - 1) / gc, 1, page_size, window, sink, splits, -1, scale, softcap, slopes,
                bias, bias_len, 0, 0, block, gate, gate_stride, gate_scale};
    for (int sh = 0; sh < 20; ++sh)
        if (page_size == 1 << sh) gm.page_shift = sh;
    cudaStream_t s = (cudaStream_t)stream;
#define RI_GO(TO, VIK, BIAS, LOW) launch_single<TO, VIK, BIAS, LOW>(q, q_stride, out, out_stride, cache, block_table, table_stride, cu_q, \
                                      kv_len, entry_list, zeros, n_entries, sink_values, part, gm, s)
#define RI_GO_L(TO, VIK, BIAS) (G <= 8 ? RI_GO(TO, VIK, BIAS, true) : RI_GO(TO, VIK, BIAS, false))
    if (value_in_key) {
        if constexpr (VD <= HD) return out_f32 ? RI_GO_L(float, true, false) : RI_GO_L(bf16, true, false);
        return (int)cudaErrorInvalidValue;
    }
    if (bias) return out_f32 ? RI_GO_L(float, false, true) : RI_GO_L(bf16, false, true);
    return out_f32 ? RI_GO_L(float, false, false) : RI_GO_L(bf16, false, false);
#undef RI_GO_L
#undef RI_GO
}

RI_API void ri_set_pdl(int on) { ri_pdl_flag() = on ? 1 : 0; }
