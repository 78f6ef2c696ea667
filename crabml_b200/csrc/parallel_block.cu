// parallel_block.cu -- the two products of a layer whose sublayers stand side by side on one norm, each fused with what surrounds it:
//
//   cc_layer_norm_product        out = W LN(x): the norm is taken while the product's operand is made, so the normed rows never exist in memory
//                                as 32-bit floats.
//   cc_joined_product_accumulate x += [W_a | W_b] [a ; glu(g, u)]: the output projections of mixer and feed-forward as ONE product over the
//                                mixer's result and the gated units, which are computed while the operand is made; the residual sum is the
//                                product's epilogue.
//
// Three forms, chosen like those of the plain product (dense.cu):
//   fewer than 8 rows            pb_matvec_kernel: every CTA stages the operand row in shared memory (norm or gated units included) and streams
//                                its weight rows past it
//   BF16, 32 rows or more, columns a multiple of 64: a kernel writes the bfloat16 operand straight from the 32-bit inputs, then the tensor-core product
//   everything else              a 32-bit operand in scratch, then the SIMT tiles
// BF16 matrices: the operand is rounded to bfloat16 once, products are exact, sums are 32-bit; F32 matrices: everything is 32-bit.
#include <cuda_bf16.h>

#include "../../include/crabml_seqops.h"
#include "act.cuh"
#include "capi_checks.cuh"
#include "layer_norm.cuh"

bool cc_prefill_bf16_supported(int64_t m, int64_t k, int64_t b);                                                                                              // prefill_gemm.cu
int cc_prefill_bf16_operand(cc_device* dev, int64_t b, int64_t k, void** out);
int cc_launch_prefill_bf16_operand(cc_device* dev, const cc_buf* w, float* out, int64_t m, int64_t k, int64_t b, int accumulate);
int cc_launch_dense_tile(cc_device* dev, const cc_buf* w, const float* x, float* out, int64_t m, int64_t k, int64_t b, int accumulate);                        // dense.cu

#define PB_THREADS 1024
#define PB_WARPS (PB_THREADS / 32)
#define PB_DEPTH 4                         // 16-byte pieces of a weight row a lane has in flight
#define PB_LN_THREADS 256

// what the operand's rows are made of
struct PbNorm {
    const float *x, *w, *b;                // x: [T, k] contiguous; b NULL: no bias
    float eps;
    __device__ __forceinline__ void stage(float* dst, int t, int k, float* red, bool round) const {
        layer_norm_row<PB_THREADS>(x + (int64_t)t * k, w, b, k, eps, red, [&](int c, float v) { dst[c] = round ? __bfloat162float(__float2bfloat16_rn(v)) : v; });
    }
};
struct PbJoin {
    const float *a, *g, *u;                // a: [T, ca] contiguous; g, u: gate and up numbers of row t at g + t * rs, u + t * rs
    int64_t rs;
    int ca, ff;
    cc_glu_params P;
    __device__ __forceinline__ float at(int t, int c) const {
        return c < ca ? a[(int64_t)t * ca + c] : glu_apply(g[t * rs + (c - ca)], u[t * rs + (c - ca)], P);
    }
    __device__ __forceinline__ void stage(float* dst, int t, int k, float*, bool round) const {
        for (int c = threadIdx.x; c < k; c += PB_THREADS) {
            const float v = at(t, c);
            dst[c] = round ? __bfloat162float(__float2bfloat16_rn(v)) : v;
        }
    }
};

__device__ __forceinline__ float pb_dot8(const int4 v, const float* a, float acc) {
    const float4 a0 = *(const float4*)a, a1 = *(const float4*)(a + 4);
    acc = fmaf(__uint_as_float((unsigned)v.x << 16), a0.x, acc); acc = fmaf(__uint_as_float((unsigned)v.x & 0xFFFF0000u), a0.y, acc);
    acc = fmaf(__uint_as_float((unsigned)v.y << 16), a0.z, acc); acc = fmaf(__uint_as_float((unsigned)v.y & 0xFFFF0000u), a0.w, acc);
    acc = fmaf(__uint_as_float((unsigned)v.z << 16), a1.x, acc); acc = fmaf(__uint_as_float((unsigned)v.z & 0xFFFF0000u), a1.y, acc);
    acc = fmaf(__uint_as_float((unsigned)v.w << 16), a1.z, acc); acc = fmaf(__uint_as_float((unsigned)v.w & 0xFFFF0000u), a1.w, acc);
    return acc;
}
// grid (about one CTA per SM, T).  `split` warps (a power of two) share one weight row, each a contiguous stretch of its 16-byte pieces in
// lane-strided order; a CTA owns PB_WARPS / split rows at a time.  A lane keeps the next PB_DEPTH pieces -- of this row or of the next one --
// in flight while it multiplies the current ones, and the first pieces are fetched before the operand row is staged.  Partial sums: the
// butterfly, then the row's warps in ascending order.  The order depends on the sizes alone, not on T.
template <bool BF16W, class Op>
__global__ void __launch_bounds__(PB_THREADS, 1) pb_matvec_kernel(const void* __restrict__ W, Op op, float* __restrict__ out, int m, int k, int split, int accumulate) {
    extern __shared__ __align__(16) float pb_sm[];              // the operand row, k floats (rounded up to 4)
    __shared__ float red[PB_WARPS];
    const int t = blockIdx.y, lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int per_cta = PB_WARPS / split, sub = warp % split, slot = warp / split;
    const int rows_it = (m + gridDim.x * per_cta - 1) / (gridDim.x * per_cta);
    const int row0 = blockIdx.x * per_cta + slot, row_step = gridDim.x * per_cta;
    float* orow = out + (int64_t)t * m;
    const bool vec = BF16W ? (k & 7) == 0 : (k & 3) == 0;
    const int pieces = BF16W ? k >> 3 : k >> 2;                  // 16-byte pieces of a row
    const int per_warp = (pieces + split - 1) / split;
    const int p_begin = min(pieces, sub * per_warp), p_end = min(pieces, p_begin + per_warp);
    const int batches = (per_warp + 32 * PB_DEPTH - 1) / (32 * PB_DEPTH);
    const int total = rows_it * batches;
    int4 cur[PB_DEPTH], nxt[PB_DEPTH];
    auto fetch = [&](int4* v, int i) {
        const int it = i / batches, p0 = p_begin + (i - it * batches) * 32 * PB_DEPTH + lane;
        const int row = row0 + it * row_step;
#pragma unroll
        for (int e = 0; e < PB_DEPTH; e++) {
            const int p = p0 + e * 32;
            v[e] = (row < m && p < p_end) ? ld_stream_16((const uint8_t*)W + ((int64_t)row * pieces + p) * 16) : make_int4(0, 0, 0, 0);
        }
    };
    if (vec) fetch(cur, 0);
    op.stage(pb_sm, t, k, red, BF16W);
    __syncthreads();
    for (int it = 0; it < rows_it; it++) {
        const int row = row0 + it * row_step;
        float acc = 0.0f;
        if (vec) {
            for (int b = 0; b < batches; b++) {
                const int i = it * batches + b;
                if (i + 1 < total) fetch(nxt, i + 1);
                const int p0 = p_begin + b * 32 * PB_DEPTH + lane;
#pragma unroll
                for (int e = 0; e < PB_DEPTH; e++) {
                    const int p = p0 + e * 32;
                    if (p < p_end) {
                        if (BF16W) acc = pb_dot8(cur[e], pb_sm + p * 8, acc);
                        else {
                            const float4 a = *(const float4*)(pb_sm + p * 4);
                            acc = fmaf(__int_as_float(cur[e].x), a.x, acc); acc = fmaf(__int_as_float(cur[e].y), a.y, acc);
                            acc = fmaf(__int_as_float(cur[e].z), a.z, acc); acc = fmaf(__int_as_float(cur[e].w), a.w, acc);
                        }
                    }
                }
#pragma unroll
                for (int e = 0; e < PB_DEPTH; e++) cur[e] = nxt[e];
            }
        } else if (row < m) {
            for (int c = sub * 32 + lane; c < k; c += split * 32)
                acc = fmaf(BF16W ? __uint_as_float((unsigned)((const uint16_t*)W)[(int64_t)row * k + c] << 16) : ((const float*)W)[(int64_t)row * k + c], pb_sm[c], acc);
        }
        acc = warp_sum(acc);
        if (split > 1) {
            __syncthreads();                                     // red may still be read
            if (lane == 0) red[warp] = acc;
            __syncthreads();
            if (sub == 0) {
                acc = 0.0f;
                for (int s = 0; s < split; s++) acc += red[warp + s];
            }
        }
        if (lane == 0 && sub == 0 && row < m) orow[row] = accumulate ? orow[row] + acc : acc;
    }
}
// the bfloat16 operand of the tensor-core product: a CTA per row
__global__ void __launch_bounds__(PB_LN_THREADS) pb_norm_bf16_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ b, __nv_bfloat16* __restrict__ out,
                                                                     int k, float eps) {
    __shared__ float red[PB_LN_THREADS / 32];
    __nv_bfloat16* o = out + (int64_t)blockIdx.x * k;
    layer_norm_row<PB_LN_THREADS>(x + (int64_t)blockIdx.x * k, w, b, k, eps, red, [&](int c, float v) { o[c] = __float2bfloat16_rn(v); });
}
__global__ void __launch_bounds__(PB_LN_THREADS) pb_norm_f32_kernel(const float* __restrict__ x, const float* __restrict__ w, const float* __restrict__ b, float* __restrict__ out, int k,
                                                                    float eps) {
    __shared__ float red[PB_LN_THREADS / 32];
    float* o = out + (int64_t)blockIdx.x * k;
    layer_norm_row<PB_LN_THREADS>(x + (int64_t)blockIdx.x * k, w, b, k, eps, red, [&](int c, float v) { o[c] = v; });
}
// grid (columns / 512, rows): two neighbouring columns per thread; k is even
__global__ void __launch_bounds__(256) pb_join_bf16_kernel(PbJoin op, __nv_bfloat16* __restrict__ out, int k) {
    const int c = (blockIdx.x * 256 + threadIdx.x) * 2, t = blockIdx.y;
    if (c < k) *(__nv_bfloat162*)(out + (int64_t)t * k + c) = __floats2bfloat162_rn(op.at(t, c), op.at(t, c + 1));
}
__global__ void __launch_bounds__(256) pb_join_f32_kernel(PbJoin op, float* __restrict__ out, int k) {
    const int c = blockIdx.x * 256 + threadIdx.x, t = blockIdx.y;
    if (c < k) out[(int64_t)t * k + c] = op.at(t, c);
}

static const size_t PB_MAX_SMEM = 200 * 1024;
static bool pb_few(int64_t T, int64_t k) { return T < 8 && (size_t)((k + 3) & ~3) * 4 <= PB_MAX_SMEM; }
template <bool BF16W, class Op>
static int pb_launch_matvec(cc_device* dev, const cc_buf* w, const Op& op, float* out, int64_t m, int64_t k, int64_t T, int accumulate) {
    const size_t smem = (size_t)((k + 3) & ~3) * 4;
    if (smem > 40 * 1024) CC_CUDA(dev, cudaFuncSetAttribute(pb_matvec_kernel<BF16W, Op>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem));
    int split = 1;                                               // as many warps per row as there are too few rows for the device's warps
    while (split < PB_WARPS && m * split * 2 <= (int64_t)dev->sm_count * PB_WARPS) split *= 2;
    const int64_t per_cta = PB_WARPS / split, ctas = (m + per_cta - 1) / per_cta;
    pb_matvec_kernel<BF16W, Op><<<dim3((unsigned)(ctas < dev->sm_count ? ctas : dev->sm_count), (unsigned)T), PB_THREADS, smem, dev->stream>>>(w->plane[0], op, out, (int)m, (int)k, split, accumulate);
    CC_LAUNCH_CHECK(dev);
    return CC_OK;
}
static bool pb_tensor_cores(const cc_buf* w, int64_t m, int64_t k, int64_t T) {
    return w->dtype == CC_BF16 && cc_prefill_bf16_supported(m, k, T) && ((uintptr_t)w->plane[0] & 15) == 0;
}

#define PB_ENTER(dev, what)                                                                                           \
    if (!(dev)) return CC_ERR_ARG;                                                                                    \
    CC_ENTER(dev);                                                                                                    \
    if (LAZY(dev)) return cc_fail((dev), CC_ERR_UNSUPPORTED, "%s: not available on a lazy (graph / megakernel) device", what)
#define PB_VIEW(dev, v, what)                                                                                         \
    do {                                                                                                              \
        if (!view_ok(v)) return cc_fail((dev), CC_ERR_ARG, "%s: bad tensor view", what);                              \
        if (!view_in_bounds(v)) return cc_fail((dev), CC_ERR_TENSOR, "%s: view addresses element %lld of a buffer of %lld", what, \
                                               (long long)view_max_offset(v), (long long)(v)->buf->nelems);           \
    } while (0)
#define PB_F32(dev, v, what)                                                        \
    do {                                                                            \
        PB_VIEW(dev, v, what);                                                      \
        REQUIRE_F32(dev, v, what);                                                  \
        CC_REQUIRE(dev, view_contiguous(v), "%s: not contiguous", what);            \
    } while (0)
#define PB_MATRIX(dev, v, what)                                                                                                                            \
    do {                                                                                                                                                   \
        PB_VIEW(dev, v, what);                                                                                                                             \
        CC_REQUIRE(dev, (v)->ndim == 2 && view_contiguous(v) && ((v)->buf->dtype == CC_F32 || (v)->buf->dtype == CC_BF16), "%s: an F32 or BF16 matrix is needed", what); \
    } while (0)
static inline const float* pb_ptr(const cc_view* v) { return (const float*)v->buf->plane[0]; }

extern "C" CC_API int cc_layer_norm_product(cc_device* dev, const cc_view* x, const cc_view* norm_w, const cc_view* norm_b, float eps, const cc_view* w, cc_buf** out) {
    PB_ENTER(dev, "layer_norm_product");
    if (!out) return cc_fail(dev, CC_ERR_ARG, "layer_norm_product: out is NULL");
    PB_F32(dev, x, "layer_norm_product x"); PB_F32(dev, norm_w, "layer_norm_product norm_w"); PB_MATRIX(dev, w, "layer_norm_product w");
    if (norm_b) PB_F32(dev, norm_b, "layer_norm_product norm_b");
    CC_REQUIRE(dev, x->ndim == 2 && x->shape[1] >= 1 && w->shape[1] == x->shape[1] && view_len(norm_w) == x->shape[1] && (!norm_b || view_len(norm_b) == x->shape[1]),
               "layer_norm_product: x must be [T, k], the norm's weight (and bias) [k] and w [m, k]");
    const int64_t T = x->shape[0], k = x->shape[1], m = w->shape[0];
    cc_buf* o = nullptr;
    int rc = cc_new_activation(dev, T * m, CC_F32, false, &o);
    if (rc) return rc;
    *out = o;
    if (T == 0 || m == 0) return CC_OK;
    const float *xp = pb_ptr(x), *nw = pb_ptr(norm_w), *nb = norm_b ? pb_ptr(norm_b) : nullptr;
    if (pb_few(T, k)) {
        const PbNorm op = {xp, nw, nb, eps};
        return w->buf->dtype == CC_BF16 ? pb_launch_matvec<true>(dev, w->buf, op, (float*)o->base, m, k, T, 0) : pb_launch_matvec<false>(dev, w->buf, op, (float*)o->base, m, k, T, 0);
    }
    if (pb_tensor_cores(w->buf, m, k, T)) {
        void* operand = nullptr;
        rc = cc_prefill_bf16_operand(dev, T, k, &operand);
        if (rc) return rc;
        pb_norm_bf16_kernel<<<(unsigned)T, PB_LN_THREADS, 0, dev->stream>>>(xp, nw, nb, (__nv_bfloat16*)operand, (int)k, eps);
        CC_LAUNCH_CHECK(dev);
        return cc_launch_prefill_bf16_operand(dev, w->buf, (float*)o->base, m, k, T, 0);
    }
    void* h = nullptr; size_t cls = 0;
    rc = cc_pool_alloc(dev, (size_t)T * k * 4, &h, &cls);
    if (rc) return rc;
    pb_norm_f32_kernel<<<(unsigned)T, PB_LN_THREADS, 0, dev->stream>>>(xp, nw, nb, (float*)h, (int)k, eps);
    dev->launches++;
    rc = cc_launch_dense_tile(dev, w->buf, (const float*)h, (float*)o->base, m, k, T, 0);
    cc_pool_free(dev, h, cls);
    return rc;
}

extern "C" CC_API int cc_joined_product_accumulate(cc_device* dev, const cc_view* dst, const cc_view* w, const cc_view* a, const cc_view* src, int32_t gate_col0, int32_t up_col0, int32_t ff,
                                                   const cc_glu_params* glu) {
    PB_ENTER(dev, "joined_product_accumulate");
    PB_F32(dev, dst, "joined_product_accumulate dst"); PB_MATRIX(dev, w, "joined_product_accumulate w"); PB_F32(dev, a, "joined_product_accumulate a");
    CC_REQUIRE(dev, dst->ndim == 2 && a->ndim == 2 && a->shape[0] == dst->shape[0] && ff >= 0 && w->shape[0] == dst->shape[1] && w->shape[1] == a->shape[1] + ff,
               "joined_product_accumulate: dst must be [T, m], a [T, ca] and w [m, ca + ff]");
    const int64_t T = dst->shape[0], m = dst->shape[1], k = w->shape[1];
    PbJoin op{};
    op.a = pb_ptr(a); op.ca = (int)a->shape[1]; op.ff = ff;
    if (ff > 0) {
        if (!src || !glu) return cc_fail(dev, CC_ERR_ARG, "joined_product_accumulate: the gated units need their numbers and constants");
        PB_VIEW(dev, src, "joined_product_accumulate src");
        REQUIRE_F32(dev, src, "joined_product_accumulate src");
        CC_REQUIRE(dev, src->ndim == 2 && src->strides[1] == 1 && src->strides[0] >= src->shape[1] && src->shape[0] == T && gate_col0 >= 0 && up_col0 >= 0 &&
                            (int64_t)gate_col0 + ff <= src->shape[1] && (int64_t)up_col0 + ff <= src->shape[1],
                   "joined_product_accumulate: src needs %d columns from columns %d and %d on", ff, gate_col0, up_col0);
        op.g = pb_ptr(src) + gate_col0; op.u = pb_ptr(src) + up_col0; op.rs = src->strides[0]; op.P = *glu;
    }
    if (T == 0 || m == 0) return CC_OK;
    float* out = (float*)dst->buf->plane[0];
    if (pb_few(T, k)) return w->buf->dtype == CC_BF16 ? pb_launch_matvec<true>(dev, w->buf, op, out, m, k, T, 1) : pb_launch_matvec<false>(dev, w->buf, op, out, m, k, T, 1);
    CC_REQUIRE(dev, T <= 65535, "joined_product_accumulate: %lld rows are too many for one pass", (long long)T);
    if (pb_tensor_cores(w->buf, m, k, T)) {
        void* operand = nullptr;
        int rc = cc_prefill_bf16_operand(dev, T, k, &operand);
        if (rc) return rc;
        pb_join_bf16_kernel<<<dim3((unsigned)((k / 2 + 255) / 256), (unsigned)T), 256, 0, dev->stream>>>(op, (__nv_bfloat16*)operand, (int)k);
        CC_LAUNCH_CHECK(dev);
        return cc_launch_prefill_bf16_operand(dev, w->buf, out, m, k, T, 1);
    }
    void* h = nullptr; size_t cls = 0;
    int rc = cc_pool_alloc(dev, (size_t)T * k * 4, &h, &cls);
    if (rc) return rc;
    pb_join_f32_kernel<<<dim3((unsigned)((k + 255) / 256), (unsigned)T), 256, 0, dev->stream>>>(op, (float*)h, (int)k);
    dev->launches++;
    rc = cc_launch_dense_tile(dev, w->buf, (const float*)h, out, m, k, T, 1);
    cc_pool_free(dev, h, cls);
    return rc;
}
