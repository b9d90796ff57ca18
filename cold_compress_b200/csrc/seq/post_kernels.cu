// post_kernels.cu -- sequence kernels, fifth part of include/cc_b200_seq.h: sublayers whose output is RMS-normed before
// it joins the residual stream, with the weighted sum over a token's experts and the copy for the next product folded in.
//
// Arithmetic rule (as in seq_kernels.cu): the stream, the expert sum and the norms are fp32 whatever the storage type.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "../../../include/cc_b200_seq.h"

namespace ccs {
int fail(int code, const char* msg);
int cuda_check(const char* where);
}  // namespace ccs

namespace ccq {
using ccs::cuda_check;
using ccs::fail;

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}
// Sum over the block in a fixed order (warp shuffles, then the warps' partial sums one after another).
__device__ __forceinline__ float block_sum(float v, float* red) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nw = (blockDim.x + 31) >> 5;
    v = warp_sum(v);
    __syncthreads();
    if (lane == 0) red[warp] = v;
    __syncthreads();
    float s = 0.f;
    for (int i = 0; i < nw; ++i) s += red[i];
    return s;
}

__device__ __forceinline__ float ldf(const float* p, int i) { return p[i]; }
__device__ __forceinline__ float ldf(const bf16* p, int i) { return __bfloat162float(p[i]); }
__device__ __forceinline__ float round_to(float v, const float*) { return v; }
__device__ __forceinline__ float round_to(float v, const bf16*) { return __bfloat162float(__float2bfloat16_rn(v)); }

// VEC consecutive floats, moved as one access when VEC is 4.
template <int VEC>
struct Pack { float v[VEC]; };
template <int VEC>
__device__ __forceinline__ Pack<VEC> load(const float* p) {
    Pack<VEC> r;
    if constexpr (VEC == 4) { const float4 f = *reinterpret_cast<const float4*>(p); r.v[0] = f.x; r.v[1] = f.y; r.v[2] = f.z; r.v[3] = f.w; }
    else r.v[0] = *p;
    return r;
}
template <int VEC>
__device__ __forceinline__ void store(float* p, const Pack<VEC>& a) {
    if constexpr (VEC == 4) *reinterpret_cast<float4*>(p) = make_float4(a.v[0], a.v[1], a.v[2], a.v[3]);
    else *p = a.v[0];
}
template <int VEC>
__device__ __forceinline__ void store(bf16* p, const Pack<VEC>& a) {
    if constexpr (VEC == 4) {
        const __nv_bfloat162 lo = __floats2bfloat162_rn(a.v[0], a.v[1]), hi = __floats2bfloat162_rn(a.v[2], a.v[3]);
        uint2 u;
        u.x = *reinterpret_cast<const uint32_t*>(&lo);
        u.y = *reinterpret_cast<const uint32_t*>(&hi);
        *reinterpret_cast<uint2*>(p) = u;
    } else *p = __float2bfloat16_rn(a.v[0]);
}

// The sublayer's row t (or the weighted sum of its experts' rows) into shared memory; returns this thread's part of its
// sum of squares.
template <int VEC>
__device__ __forceinline__ float sublayer_row(const CcSeqPostNorm& a, size_t t, float* row, int tid, int step) {
    const int E = a.E;
    float ss = 0.f;
    for (int e = tid * VEC; e < E; e += step) {
        Pack<VEC> r;
        if (a.top == 0) {
            r = load<VEC>(a.y + t * a.ldy + e);
        } else {
#pragma unroll
            for (int i = 0; i < VEC; ++i) r.v[i] = 0.f;
            for (int k = 0; k < a.top; ++k) {
                const size_t m = t * a.top + k;
                const float w = a.wts[m];
                const Pack<VEC> y = load<VEC>(a.y + (a.slot != nullptr ? (size_t)a.slot[m] : m) * E + e);
#pragma unroll
                for (int i = 0; i < VEC; ++i) r.v[i] = fmaf(w, y.v[i], r.v[i]);
            }
        }
        store<VEC>(row + e, r);
#pragma unroll
        for (int i = 0; i < VEC; ++i) ss = fmaf(r.v[i], r.v[i], ss);
    }
    return ss;
}

// One CTA per row.  The sublayer's row (or the weighted sum of its experts' rows) is read once into shared memory with
// its sum of squares; the second pass adds the normed row to the stream; with a following norm the sum stays in shared
// memory for a third pass.  Every pass is a chain of dependent loads, so a step of few rows runs up to 1024 threads per
// row and a long one 256 (more rows per SM).
template <typename AT, int VEC>
__global__ void __launch_bounds__(1024) post_norm_kernel(const CcSeqPostNorm a) {
    extern __shared__ float4 pn4[];
    float* row = reinterpret_cast<float*>(pn4);        // [E]
    __shared__ float red[32];
    const int E = a.E, tid = threadIdx.x, step = blockDim.x * VEC;
    const size_t t = blockIdx.x, base = t * E;
    float ss = sublayer_row<VEC>(a, t, row, tid, step);
    const float rinv = 1.0f / sqrtf(block_sum(ss, red) / (float)E + a.eps);
    AT* act = (AT*)a.x_act;
    float* out = a.x_out != nullptr ? a.x_out : a.x;
    ss = 0.f;
    for (int e = tid * VEC; e < E; e += step) {
        Pack<VEC> s = load<VEC>(a.x + base + e);
        const Pack<VEC> r = load<VEC>(row + e), w = load<VEC>(a.w + e);
#pragma unroll
        for (int i = 0; i < VEC; ++i) s.v[i] += r.v[i] * rinv * (w.v[i] + a.gain_offset);
        store<VEC>(out + base + e, s);
        if (a.next_w == nullptr) {
            if (act != nullptr) store<VEC>(act + base + e, s);
        } else {
            store<VEC>(row + e, s);
#pragma unroll
            for (int i = 0; i < VEC; ++i) ss = fmaf(s.v[i], s.v[i], ss);
        }
    }
    if (a.next_w == nullptr || act == nullptr) return;
    const float rnext = 1.0f / sqrtf(block_sum(ss, red) / (float)E + a.next_eps);
    for (int e = tid * VEC; e < E; e += step) {
        Pack<VEC> s = load<VEC>(row + e);
        const Pack<VEC> w = load<VEC>(a.next_w + e);
#pragma unroll
        for (int i = 0; i < VEC; ++i) s.v[i] = s.v[i] * rnext * (w.v[i] + a.next_offset);
        store<VEC>(act + base + e, s);
    }
}

// The same sum for one token of a step of few, then the router of the feed-forward that reads it: a warp per expert row
// against the sum in shared memory (rounded as the product's input is), then one warp takes the `top` largest logits and
// their softmax.
template <typename AT, int VEC>
__global__ void __launch_bounds__(1024) post_norm_route_kernel(const CcSeqPostNorm a, const AT* __restrict__ Wr, const float* __restrict__ bias,
                                                               int n, int top, int32_t* __restrict__ ids, float* __restrict__ wts) {
    extern __shared__ float4 pn4[];
    float* row = reinterpret_cast<float*>(pn4);        // [E]
    float* z = row + ((a.E + 3) & ~3);                 // [n]
    __shared__ float red[32];
    const int E = a.E, tid = threadIdx.x, step = blockDim.x * VEC, lane = tid & 31, warp = tid >> 5, nw = blockDim.x >> 5;
    const size_t t = blockIdx.x, base = t * E;
    const float ss = sublayer_row<VEC>(a, t, row, tid, step);
    const float rinv = 1.0f / sqrtf(block_sum(ss, red) / (float)E + a.eps);
    AT* act = (AT*)a.x_act;
    float* out = a.x_out != nullptr ? a.x_out : a.x;
    for (int e = tid * VEC; e < E; e += step) {
        Pack<VEC> s = load<VEC>(a.x + base + e);
        const Pack<VEC> r = load<VEC>(row + e), w = load<VEC>(a.w + e);
#pragma unroll
        for (int i = 0; i < VEC; ++i) s.v[i] += r.v[i] * rinv * (w.v[i] + a.gain_offset);
        store<VEC>(out + base + e, s);
        if (act != nullptr) store<VEC>(act + base + e, s);
#pragma unroll
        for (int i = 0; i < VEC; ++i) s.v[i] = round_to(s.v[i], Wr);
        store<VEC>(row + e, s);
    }
    __syncthreads();
    constexpr int W16 = 16 / (int)sizeof(AT);
    for (int i = warp; i < n; i += nw) {
        const AT* w = Wr + (size_t)i * E;
        float acc = 0.f;
        if (E % W16 == 0) {
            const uint4* w16 = reinterpret_cast<const uint4*>(w);
#pragma unroll 8
            for (int c = lane; c < E / W16; c += 32) {
                const uint4 u = __ldg(w16 + c);
                const AT* e = reinterpret_cast<const AT*>(&u);
                const float4* x4 = reinterpret_cast<const float4*>(row + c * W16);
#pragma unroll
                for (int q = 0; q < W16 / 4; ++q) {
                    const float4 xv = x4[q];
                    acc = fmaf(ldf(e, 4 * q + 0), xv.x, acc);
                    acc = fmaf(ldf(e, 4 * q + 1), xv.y, acc);
                    acc = fmaf(ldf(e, 4 * q + 2), xv.z, acc);
                    acc = fmaf(ldf(e, 4 * q + 3), xv.w, acc);
                }
            }
        } else {
            for (int e = lane; e < E; e += 32) acc = fmaf(ldf(w, e), row[e], acc);
        }
        acc = warp_sum(acc);
        if (lane == 0) z[i] = acc + (bias != nullptr ? bias[i] : 0.f);
    }
    __syncthreads();
    if (warp != 0) return;
    float sum = 0.f, z0 = 0.f;
    for (int k = 0; k < top; ++k) {
        float bv = -INFINITY;
        int bi = 0x7fffffff;
        for (int i = lane; i < n; i += 32) {
            const float v = z[i];
            if (v > bv) { bv = v; bi = i; }
        }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ov = __shfl_xor_sync(0xffffffffu, bv, o);
            const int oi = __shfl_xor_sync(0xffffffffu, bi, o);
            if (ov > bv || (ov == bv && oi < bi)) { bv = ov; bi = oi; }
        }
        if (bi >= n) bi = 0;   // logits that are not numbers: kept harmless
        if (k == 0) z0 = bv;
        const float w = expf(bv - z0);
        sum += w;
        if (lane == 0) {
            ids[t * top + k] = bi;
            wts[t * top + k] = w;
            z[bi] = -INFINITY;
        }
        __syncwarp();
    }
    for (int k = lane; k < top; k += 32) wts[t * top + k] /= sum;
}

template <typename K>
static int more_smem(K kern, size_t smem, size_t& configured) {
    if (smem <= configured) return CC_SEQ_OK;
    if (cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess) return cuda_check("post_norm: shared memory");
    configured = smem;
    return CC_SEQ_OK;
}

template <typename AT, int VEC>
static int launch_post_norm(const CcSeqPostNorm* a, cudaStream_t st) {
    const size_t smem = sizeof(float) * (size_t)((a->E + 3) & ~3);
    static size_t configured = 48 * 1024;
    auto kern = post_norm_kernel<AT, VEC>;
    if (int rc = more_smem(kern, smem, configured)) return rc;
    const int want = ((a->E + VEC - 1) / VEC + 31) / 32 * 32, most = a->T < 64 ? 1024 : 256;
    kern<<<a->T, want < most ? want : most, smem, st>>>(*a);
    return cuda_check("post_norm_kernel");
}

template <typename AT, int VEC>
static int launch_post_norm_route(const CcSeqPostNorm* a, const void* Wr, const float* bias, int n, int top, int32_t* ids, float* wts, cudaStream_t st) {
    const size_t smem = sizeof(float) * (size_t)(((a->E + 3) & ~3) + n);
    static size_t configured = 48 * 1024;
    auto kern = post_norm_route_kernel<AT, VEC>;
    if (int rc = more_smem(kern, smem, configured)) return rc;
    int threads = ((a->E + VEC - 1) / VEC + 31) / 32 * 32;
    threads = threads > n * 32 ? threads : n * 32;      // at least a warp per expert
    kern<<<a->T, threads < 1024 ? threads : 1024, smem, st>>>(*a, (const AT*)Wr, bias, n, top, ids, wts);
    return cuda_check("post_norm_route_kernel");
}

static int check_post_norm(const CcSeqPostNorm* a) {
    if (!a || !a->x || !a->y || !a->w || a->T < 1 || a->E < 1 || a->top < 0 || (a->top > 0 && !a->wts) || (a->next_w && !a->x_act))
        return fail(CC_SEQ_ERR_INVALID_ARG, "post_norm: bad argument");
    if ((size_t)a->E * 4 > 180 * 1024) return fail(CC_SEQ_ERR_UNSUPPORTED_SHAPE, "post_norm: rows longer than 46080");
    if (a->act_dtype != CC_DT_F32 && a->act_dtype != CC_DT_BF16) return fail(CC_SEQ_ERR_INVALID_ARG, "unknown element type");
    return CC_SEQ_OK;
}

static bool wide_rows(const CcSeqPostNorm* a) {
    const uintptr_t all = (uintptr_t)a->x | (uintptr_t)a->y | (uintptr_t)a->w | (uintptr_t)a->x_out | (uintptr_t)a->x_act | (uintptr_t)a->next_w;
    return a->E % 4 == 0 && a->ldy % 4 == 0 && (all & 15) == 0;
}

}  // namespace ccq

using namespace ccq;

extern "C" {

int cc_seq_post_norm(const CcSeqPostNorm* a, void* stream) {
    if (int rc = check_post_norm(a)) return rc;
    cudaStream_t st = (cudaStream_t)stream;
    const bool vec = wide_rows(a);
    if (a->act_dtype == CC_DT_BF16) return vec ? launch_post_norm<bf16, 4>(a, st) : launch_post_norm<bf16, 1>(a, st);
    return vec ? launch_post_norm<float, 4>(a, st) : launch_post_norm<float, 1>(a, st);
}

int cc_seq_post_norm_route(const CcSeqPostNorm* a, const void* Wr, const float* bias, int32_t n, int32_t top, int32_t* ids,
                           float* wts, void* stream) {
    if (int rc = check_post_norm(a)) return rc;
    if (!Wr || !ids || !wts || n < 1 || top < 1 || top > n || a->next_w || n > 4096)
        return fail(CC_SEQ_ERR_INVALID_ARG, "post_norm_route: bad argument");
    cudaStream_t st = (cudaStream_t)stream;
    const bool vec = wide_rows(a);
#define CALL(AT, VEC) launch_post_norm_route<AT, VEC>(a, Wr, bias, n, top, ids, wts, st)
    if (a->act_dtype == CC_DT_BF16) return vec ? CALL(bf16, 4) : CALL(bf16, 1);
    return vec ? CALL(float, 4) : CALL(float, 1);
#undef CALL
}

}  // extern "C"
