// cell_kernels.cu -- sequence kernels, sixth part of include/cc_b200_seq.h: element-wise bounded norms around every
// sublayer (the residual sum, the norm of the sublayer's result and the next sublayer's norm are one pass), and the matrix
// memory with exponential gates, token by token for short steps and in chunks for long ones.
//
// Arithmetic rule (as in seq_kernels.cu): the stream, the norms, gates, decays and the whole recurrence are fp32 whatever
// the storage type; expf / tanhf / log1pf are the accurate versions.  Sums of log gates over many tokens, of which only
// differences are used, are kept in fp64.
#include <cuda_bf16.h>
#include <cuda_runtime.h>
#include <math.h>
#include <stdint.h>

#include "../../../include/cc_b200_seq.h"

namespace ccs {
int fail(int code, const char* msg);
int cuda_check(const char* where);
}  // namespace ccs

namespace ccc {
using ccs::cuda_check;
using ccs::fail;

typedef __nv_bfloat16 bf16;

__device__ __forceinline__ float ldf(const float* p, size_t i) { return p[i]; }
__device__ __forceinline__ float ldf(const bf16* p, size_t i) { return __bfloat162float(p[i]); }

__device__ __forceinline__ float warp_sum(float v) {
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) v += __shfl_xor_sync(0xffffffffu, v, o);
    return v;
}

// VEC consecutive values, moved as one access when VEC is 4.
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
__device__ __forceinline__ Pack<VEC> load(const bf16* p) {
    Pack<VEC> r;
    if constexpr (VEC == 4) {
        const uint2 u = *reinterpret_cast<const uint2*>(p);
        const bf16* e = reinterpret_cast<const bf16*>(&u);
#pragma unroll
        for (int i = 0; i < 4; ++i) r.v[i] = __bfloat162float(e[i]);
    } else r.v[0] = __bfloat162float(*p);
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

// ------------------------------------------------------------------------------------------------ bounded norms
// A norm's parameters for the VEC channels a thread owns, read once and used for every row it walks.
template <int VEC>
struct Bounded {
    float alpha;
    Pack<VEC> w, b;
    __device__ __forceinline__ Bounded(const CcSeqBounded& p, int c) {
        if (p.w == nullptr) return;
        alpha = *p.alpha;
        w = load<VEC>(p.w + c);
        b = load<VEC>(p.b + c);
    }
    __device__ __forceinline__ float operator()(float v, int i) const { return fmaf(w.v[i], tanhf(alpha * v), b.v[i]); }
};

template <typename AT, int VEC>
__global__ void __launch_bounds__(128) bounded_sum_kernel(const CcSeqBoundedSum a) {
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC, E = a.E;
    if (c >= E) return;
    const Bounded<VEC> out(a.out_norm, c), next(a.next_norm, c);
    for (int t = blockIdx.y; t < a.T; t += gridDim.y) {
        const size_t src = a.rows != nullptr ? (size_t)a.rows[t] : (size_t)t, dst = (size_t)t * E + c;
        Pack<VEC> s = load<VEC>(a.x + src * E + c);
        if (a.y != nullptr) {
            const Pack<VEC> y = load<VEC>(a.y + src * a.ldy + c);
#pragma unroll
            for (int i = 0; i < VEC; ++i) s.v[i] = fmaf(a.mult, out(y.v[i], i), s.v[i]);
        }
        if (a.add != nullptr) {
            const Pack<VEC> d = load<VEC>(a.add + src * E + c);
#pragma unroll
            for (int i = 0; i < VEC; ++i) s.v[i] += d.v[i];
        }
        if (a.x_out != nullptr) store<VEC>(a.x_out + dst, s);
        if (a.h != nullptr) {
#pragma unroll
            for (int i = 0; i < VEC; ++i) s.v[i] = next(s.v[i], i);
            store<VEC>((AT*)a.h + dst, s);
        }
    }
}

template <typename ST, typename AT, int VEC>
__global__ void __launch_bounds__(128) embed_bounded_kernel(const int32_t* __restrict__ tokens, const ST* __restrict__ embed, const CcSeqBounded emb_p,
                                                            float* __restrict__ x, const CcSeqBounded next_p, AT* __restrict__ h, int T, int E) {
    const int c = (blockIdx.x * blockDim.x + threadIdx.x) * VEC;
    if (c >= E) return;
    const Bounded<VEC> emb(emb_p, c), next(next_p, c);
    for (int t = blockIdx.y; t < T; t += gridDim.y) {
        Pack<VEC> s = load<VEC>(embed + (size_t)tokens[t] * E + c);
#pragma unroll
        for (int i = 0; i < VEC; ++i) s.v[i] = emb(s.v[i], i);
        store<VEC>(x + (size_t)t * E + c, s);
        if (h == nullptr) continue;
#pragma unroll
        for (int i = 0; i < VEC; ++i) s.v[i] = next(s.v[i], i);
        store<VEC>(h + (size_t)t * E + c, s);
    }
}

// columns x rows: a thread keeps its channels' parameters over several rows once the GPU is filled
static dim3 row_grid(int T, int E, int vec) {
    const int cols = (E + 128 * vec - 1) / (128 * vec), want = (148 * 16 + cols - 1) / cols;
    return dim3(cols, T < want ? T : want);
}

// ------------------------------------------------------------------------------------------------ matrix memory: gates
__device__ __forceinline__ float input_gate(float raw, float bias, float cap) { return cap * tanhf((raw + bias) / cap); }
__device__ __forceinline__ float forget_gate(float raw, float bias, float cap) {
    const float z = cap * tanhf((raw + bias) / cap);
    return fminf(z, 0.f) - log1pf(expf(-fabsf(z)));
}

// ------------------------------------------------------------------------------------------------ matrix memory: scan
// CTA = one head x 32 value columns; warp p keeps state rows p * CH .. of its lane's column in registers, one more warp
// keeps the key sum.  Per batch of TB tokens: the rows are staged (k times its gate), the running maximum is walked, the
// warps run the tokens independently of one another, and the read-outs (summed in warp order) meet their denominators.
// Every CTA of a head carries the key sum and the maximum; the last one to finish writes them back (the counter behind
// the maximum is zero between calls), so no CTA can still be reading them.
constexpr int SCAN_J = 32, SCAN_TB = 16, SCAN_ND = 16;   // key-sum entries per lane: heads of up to 512

template <int CH>
__global__ void __launch_bounds__(544) mlstm_scan_kernel(const CcSeqMlstm a) {
    extern __shared__ float4 ml4[];
    __shared__ float s_i[SCAN_TB], s_f[SCAN_TB], s_m[SCAN_TB + 1], s_keep[SCAN_TB], s_floor[SCAN_TB], s_den[SCAN_TB];
    __shared__ int s_last;
    const int D = a.D, P = (D + CH - 1) / CH, Dp = P * CH, TB = min(a.T, SCAN_TB);
    float* qs = reinterpret_cast<float*>(ml4);      // [TB][Dp]
    float* ks = qs + TB * Dp;                       // [TB][Dp]
    float* vs = ks + TB * Dp;                       // [TB][32]
    float* part = vs + TB * SCAN_J;                 // [TB][P][32]
    const int h = blockIdx.x, j0 = blockIdx.y * SCAN_J;
    const int tid = threadIdx.x, nth = blockDim.x, lane = tid & 31, p = tid >> 5, j = j0 + lane, n0 = p * CH;
    float* S = a.state + (size_t)h * D * a.V;
    float* aux = a.aux + (size_t)h * (D + 2);
    const bool columns = p < P;
    float st[CH], ns[SCAN_ND];
    if (columns) {
#pragma unroll
        for (int c = 0; c < CH; ++c) st[c] = (n0 + c < D && j < a.V) ? S[(size_t)(n0 + c) * a.V + j] : 0.f;
    } else {
#pragma unroll
        for (int i = 0; i < SCAN_ND; ++i) ns[i] = lane + 32 * i < D ? aux[lane + 32 * i] : 0.f;
    }
    if (tid == 0) s_m[0] = aux[D];
    const float ib = a.i_bias[h], fb = a.f_bias[h];
    for (int tb = 0; tb < a.T; tb += TB) {
        const int nt = min(TB, a.T - tb);
        for (int idx = tid; idx < nt * Dp; idx += nth) {
            const int t = idx / Dp, d = idx - t * Dp;
            const size_t o = (size_t)(tb + t) * a.ld + (size_t)h * D + d;
            qs[idx] = d < D ? a.q[o] * a.q_scale : 0.f;
            ks[idx] = d < D ? a.k[o] : 0.f;
        }
        for (int idx = tid; idx < nt * SCAN_J; idx += nth) {
            const int t = idx / SCAN_J, c = idx - t * SCAN_J;
            vs[idx] = j0 + c < a.V ? a.v[(size_t)(tb + t) * a.ld + (size_t)h * a.V + j0 + c] : 0.f;
        }
        if (tid < nt) {
            s_i[tid] = input_gate(a.i_raw[(size_t)(tb + tid) * a.ld + h], ib, a.gate_cap);
            s_f[tid] = forget_gate(a.f_raw[(size_t)(tb + tid) * a.ld + h], fb, a.gate_cap);
        }
        __syncthreads();
        if (tid == 0)
            for (int t = 0; t < nt; ++t) s_m[t + 1] = fmaxf(s_f[t] + s_m[t], s_i[t]);
        __syncthreads();
        if (tid < nt) {
            s_keep[tid] = expf(s_f[tid] + s_m[tid] - s_m[tid + 1]);
            s_i[tid] = expf(s_i[tid] - s_m[tid + 1]);
            s_floor[tid] = expf(-s_m[tid + 1]);
        }
        __syncthreads();
        if (tid == 0) s_m[0] = s_m[nt];      // read again only after the next batch's first barrier
        if (columns) {
            for (int t = 0; t < nt; ++t) {
                const float keep = s_keep[t], v = vs[t * SCAN_J + lane] * s_i[t];
                const float4* q4 = reinterpret_cast<const float4*>(qs + t * Dp + n0);
                const float4* k4 = reinterpret_cast<const float4*>(ks + t * Dp + n0);
                float acc = 0.f;
#pragma unroll
                for (int c4 = 0; c4 < CH / 4; ++c4) {
                    const float4 qv = q4[c4], kv = k4[c4];
                    const float q_[4] = {qv.x, qv.y, qv.z, qv.w}, k_[4] = {kv.x, kv.y, kv.z, kv.w};
#pragma unroll
                    for (int i = 0; i < 4; ++i) {
                        st[4 * c4 + i] = fmaf(keep, st[4 * c4 + i], k_[i] * v);
                        acc = fmaf(q_[i], st[4 * c4 + i], acc);
                    }
                }
                part[(t * P + p) * SCAN_J + lane] = acc;
            }
        } else {
            for (int t = 0; t < nt; ++t) {
                const float keep = s_keep[t], add = s_i[t];
                float acc = 0.f;
#pragma unroll
                for (int i = 0; i < SCAN_ND; ++i) {
                    const int d = lane + 32 * i;
                    if (d < D) {
                        ns[i] = fmaf(keep, ns[i], add * ks[t * Dp + d]);
                        acc = fmaf(qs[t * Dp + d], ns[i], acc);
                    }
                }
                acc = warp_sum(acc);
                if (lane == 0) s_den[t] = fmaxf(fabsf(acc), s_floor[t]) + a.den_eps;
            }
        }
        __syncthreads();
        for (int idx = tid; idx < nt * SCAN_J; idx += nth) {
            const int t = idx / SCAN_J, c = idx - t * SCAN_J;
            if (j0 + c >= a.V) continue;
            float o = 0.f;
            for (int w = 0; w < P; ++w) o += part[(t * P + w) * SCAN_J + c];
            a.o[(size_t)(tb + t) * a.H * a.V + (size_t)h * a.V + j0 + c] = o / s_den[t];
        }
        __syncthreads();
    }
    if (columns) {
#pragma unroll
        for (int c = 0; c < CH; ++c)
            if (n0 + c < D && j < a.V) S[(size_t)(n0 + c) * a.V + j] = st[c];
    }
    if (tid == 0) s_last = atomicAdd((int*)(aux + D + 1), 1) == (int)gridDim.y - 1;
    __syncthreads();
    if (!s_last) return;
    if (!columns) {
#pragma unroll
        for (int i = 0; i < SCAN_ND; ++i)
            if (lane + 32 * i < D) aux[lane + 32 * i] = ns[i];
    }
    if (tid == 0) {
        aux[D] = s_m[0];
        *(int*)(aux + D + 1) = 0;
    }
}

// ------------------------------------------------------------------------------------------------ matrix memory: chunks
// With F_t = sum of the log forget gates of tokens 1 .. t (F_0 = 0) and m_0 the carried maximum, unrolling the recurrence
// gives  m_t = F_t + max(m_0, max_{s <= t} (i_s - F_s))  and the weight of token s in the state after token t as
// exp(F_t - F_s + i_s - m_t); the state at a chunk's start enters with exp(F_t - F_start + m_start - m_t).
constexpr int CK = 64;            // tokens per chunk
constexpr int CT = 64;            // state rows / value columns per tile
constexpr int GATE_TILE = 4096, GATE_THREADS = 256, GATE_PER = GATE_TILE / GATE_THREADS;

struct ChunkSpace {               // the workspace, cut up
    double* F;                    // [H][T + 1]
    float* m;                     // [H][T + 1]
    float* i;                     // [H][T]
    float* N;                     // [chunks][H][D]      the chunk's key sum, then the key sum before the chunk
    float* S;                     // [chunks][H][D][V]   the same for the state
    int chunks;
};

__host__ __device__ inline size_t up16(size_t n) { return (n + 15) & ~(size_t)15; }

__host__ __device__ inline size_t chunk_space(ChunkSpace* w, void* base, int T, int H, int D, int V) {
    const size_t chunks = (size_t)(T + CK - 1) / CK, rows = (size_t)H * (T + 1);
    size_t o = 0;
    char* b = (char*)base;
    if (w) { w->F = (double*)(b + o); w->chunks = (int)chunks; }
    o += up16(rows * sizeof(double));
    if (w) w->m = (float*)(b + o);
    o += up16(rows * sizeof(float));
    if (w) w->i = (float*)(b + o);
    o += up16((size_t)H * T * sizeof(float));
    if (w) w->N = (float*)(b + o);
    o += up16(chunks * H * D * sizeof(float));
    if (w) w->S = (float*)(b + o);
    return o + up16(chunks * H * D * V * sizeof(float));
}

// Exclusive scan over the block of one value per thread (identity e for thread 0); `total` gets the whole.
template <typename Op>
__device__ __forceinline__ double block_scan(double v, double e, double* red, double& total, Op op) {
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    double inc = v;
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double u = __shfl_up_sync(0xffffffffu, inc, o);
        if (lane >= o) inc = op(u, inc);
    }
    __syncthreads();
    if (lane == 31) red[warp] = inc;
    __syncthreads();
    double before = e;
    total = e;
    for (int w = 0; w < GATE_THREADS / 32; ++w) {
        if (w < warp) before = op(before, red[w]);
        total = op(total, red[w]);
    }
    const double left = __shfl_up_sync(0xffffffffu, inc, 1);
    return lane == 0 ? before : op(before, left);
}

// One CTA per head: the gates of all tokens (independent loads), then their sums and the running maximum; a thread walks
// GATE_PER consecutive tokens of the tile in shared memory.
__global__ void __launch_bounds__(GATE_THREADS) mlstm_gates_kernel(const CcSeqMlstm a, const ChunkSpace w) {
    __shared__ float si[GATE_TILE + GATE_THREADS], sf[GATE_TILE + GATE_THREADS];
    __shared__ double red[GATE_THREADS / 32];
    const int h = blockIdx.x, tid = threadIdx.x, T = a.T;
    const float ib = a.i_bias[h], fb = a.f_bias[h];
    double* F = w.F + (size_t)h * (T + 1);
    float* m = w.m + (size_t)h * (T + 1);
    float* gi = w.i + (size_t)h * T;
    const float m0 = a.aux[(size_t)h * (a.D + 2) + a.D];
    double base = 0.0, best = m0;
    if (tid == 0) { F[0] = 0.0; m[0] = m0; }
    auto at = [](int t) { return t + t / GATE_PER; };      // threads' runs start in different banks
    for (int tb = 0; tb < T; tb += GATE_TILE) {
        const int nt = min(GATE_TILE, T - tb);
        __syncthreads();
        for (int t = tid; t < nt; t += GATE_THREADS) {
            const size_t o = (size_t)(tb + t) * a.ld + h;
            const float iv = input_gate(a.i_raw[o], ib, a.gate_cap);
            si[at(t)] = iv;
            gi[tb + t] = iv;
            sf[at(t)] = forget_gate(a.f_raw[o], fb, a.gate_cap);
        }
        __syncthreads();
        const int t0 = tid * GATE_PER, t1 = min(nt, t0 + GATE_PER);
        double sum = 0.0;
        for (int t = t0; t < t1; ++t) sum += sf[at(t)];
        double all, most;
        double f = base + block_scan(sum, 0.0, red, all, [](double x, double y) { return x + y; });
        double run = f, top = -INFINITY;
        for (int t = t0; t < t1; ++t) { run += sf[at(t)]; top = fmax(top, si[at(t)] - run); }
        double b = fmax(best, block_scan(top, -INFINITY, red, most, [](double x, double y) { return fmax(x, y); }));
        for (int t = t0; t < t1; ++t) {
            f += sf[at(t)];
            b = fmax(b, si[at(t)] - f);
            F[tb + t + 1] = f;
            m[tb + t + 1] = (float)(f + b);
        }
        base += all;
        best = fmax(best, most);
    }
}

// The chunk's own sums: S_c = sum_s w_s k_s v_s^T and n_c = sum_s w_s k_s, w_s the weight of token s at the chunk's end.
// CTA = (chunk, head, tile of 64 state rows x 64 columns); thread (ty, tx) owns 4 x 4 of the tile.
__global__ void __launch_bounds__(256) mlstm_chunk_sums_kernel(const CcSeqMlstm a, const ChunkSpace w) {
    __shared__ float4 k4[CK * CT / 4], v4[CK * CT / 4];
    __shared__ float ws[CK];
    float* ks = reinterpret_cast<float*>(k4);
    float* vs = reinterpret_cast<float*>(v4);
    const int c = blockIdx.x, h = blockIdx.y, tiles_v = (a.V + CT - 1) / CT, T = a.T, D = a.D, V = a.V;
    const int d0 = (blockIdx.z / tiles_v) * CT, v0 = (blockIdx.z % tiles_v) * CT;
    const int t0 = c * CK, nt = min(CK, T - t0), tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    const double* F = w.F + (size_t)h * (T + 1);
    if (tid < CK) {
        const double end = F[t0 + nt] - (double)w.m[(size_t)h * (T + 1) + t0 + nt];
        ws[tid] = tid < nt ? expf((float)(end - F[t0 + tid + 1] + (double)w.i[(size_t)h * T + t0 + tid])) : 0.f;
    }
    __syncthreads();
#pragma unroll 4
    for (int idx = tid; idx < CK * CT; idx += 256) {
        const int t = idx / CT, x = idx % CT;
        const size_t row = (size_t)(t0 + t) * a.ld;
        ks[idx] = t < nt && d0 + x < D ? a.k[row + (size_t)h * D + d0 + x] * ws[t] : 0.f;
        vs[idx] = t < nt && v0 + x < V ? a.v[row + (size_t)h * V + v0 + x] : 0.f;
    }
    __syncthreads();
    float acc[4][4];
#pragma unroll
    for (int r = 0; r < 4; ++r)
#pragma unroll
        for (int e = 0; e < 4; ++e) acc[r][e] = 0.f;
#pragma unroll 8
    for (int s = 0; s < CK; ++s) {
        const float4 kv = k4[s * (CT / 4) + ty], vv = v4[s * (CT / 4) + tx];
        const float kr[4] = {kv.x, kv.y, kv.z, kv.w}, ve[4] = {vv.x, vv.y, vv.z, vv.w};
#pragma unroll
        for (int r = 0; r < 4; ++r)
#pragma unroll
            for (int e = 0; e < 4; ++e) acc[r][e] = fmaf(kr[r], ve[e], acc[r][e]);
    }
    float* S = w.S + ((size_t)c * a.H + h) * D * V;
#pragma unroll
    for (int r = 0; r < 4; ++r) {
        const int d = d0 + 4 * ty + r;
        if (d >= D) continue;
        if (V % 4 == 0 && v0 + 4 * tx < V) {
            *reinterpret_cast<float4*>(S + (size_t)d * V + v0 + 4 * tx) = make_float4(acc[r][0], acc[r][1], acc[r][2], acc[r][3]);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (v0 + 4 * tx + e < V) S[(size_t)d * V + v0 + 4 * tx + e] = acc[r][e];
        }
    }
    if (v0 == 0 && tid < CT && d0 + tid < D) {
        float n = 0.f;
        for (int s = 0; s < CK; ++s) n += ks[s * CT + tid];
        w.N[((size_t)c * a.H + h) * D + d0 + tid] = n;
    }
}

// Chunk after chunk, a thread per state entry (or key-sum entry): the entry's chunk sum is replaced by its value before the
// chunk; the value after the last chunk is the new state.
constexpr int PASS_CHUNKS = 256, PASS_AHEAD = 8;
__global__ void __launch_bounds__(256) mlstm_pass_kernel(const CcSeqMlstm a, const ChunkSpace w) {
    __shared__ float decay[PASS_CHUNKS];
    const int h = blockIdx.y, D = a.D, V = a.V, T = a.T, tid = threadIdx.x;
    const size_t e = (size_t)blockIdx.x * 256 + tid, DV = (size_t)D * V;
    const bool key = e >= DV, live = e < DV + D;
    float* aux = a.aux + (size_t)h * (D + 2);
    float* home = key ? aux + (e - DV) : a.state + (size_t)h * DV + e;
    float* buf = key ? w.N + (size_t)h * D + (e - DV) : w.S + (size_t)h * DV + e;
    const size_t stride = (size_t)a.H * (key ? (size_t)D : DV);
    const double* F = w.F + (size_t)h * (T + 1);
    const float* m = w.m + (size_t)h * (T + 1);
    float v = live ? *home : 0.f;
    for (int c0 = 0; c0 < w.chunks; c0 += PASS_CHUNKS) {
        const int nc = min(PASS_CHUNKS, w.chunks - c0);
        __syncthreads();
        if (tid < nc) {
            const int from = (c0 + tid) * CK, to = min(T, from + CK);
            decay[tid] = expf((float)(F[to] - F[from] + (double)m[from] - (double)m[to]));
        }
        __syncthreads();
        if (!live) continue;
        for (int c = 0; c < nc; c += PASS_AHEAD) {
            float own[PASS_AHEAD];
#pragma unroll
            for (int i = 0; i < PASS_AHEAD; ++i) own[i] = c + i < nc ? buf[(size_t)(c0 + c + i) * stride] : 0.f;
#pragma unroll
            for (int i = 0; i < PASS_AHEAD; ++i)
                if (c + i < nc) {
                    buf[(size_t)(c0 + c + i) * stride] = v;
                    v = fmaf(decay[c + i], v, own[i]);
                }
        }
    }
    if (live) *home = v;
    if (blockIdx.x == 0 && tid == 0) aux[D] = m[T];
}

// Outputs of one (chunk, head, 64 value columns): scores q k^T and read-outs of the state before the chunk accumulate
// together over slices of 32 state rows (q staged once for both); then the weighted scores meet the chunk's values.
// Thread (ty, tx) owns tokens 4 ty .. x keys 4 tx .. of the scores and tokens x columns 4 tx .. of the outputs.
constexpr int DS = 32, QP = CK + 4;
__global__ void __launch_bounds__(256) mlstm_chunk_out_kernel(const CcSeqMlstm a, const ChunkSpace w) {
    __shared__ float4 pool[2 * DS * QP / 4];       // q and k slices, transposed; later the weighted scores, transposed
    __shared__ float4 s4[DS * CT / 4], v4[CK * CT / 4];
    __shared__ double Fs[CK + 1];
    __shared__ float is[CK], ms[CK + 1], nsl[DS];
    float* qT = reinterpret_cast<float*>(pool);
    float* kT = qT + DS * QP;
    float* pT = qT;                                // [CK][QP]
    float* Ss = reinterpret_cast<float*>(s4);
    float* vs = reinterpret_cast<float*>(v4);
    const int c = blockIdx.x, h = blockIdx.y, v0 = blockIdx.z * CT, T = a.T, D = a.D, V = a.V;
    const int t0 = c * CK, nt = min(CK, T - t0), tid = threadIdx.x, tx = tid & 15, ty = tid >> 4;
    if (tid <= nt) {
        Fs[tid] = w.F[(size_t)h * (T + 1) + t0 + tid];
        ms[tid] = w.m[(size_t)h * (T + 1) + t0 + tid];
        if (tid < nt) is[tid] = w.i[(size_t)h * T + t0 + tid];
    }
#pragma unroll 4
    for (int idx = tid; idx < CK * CT; idx += 256) {
        const int t = idx / CT, x = idx % CT;
        vs[idx] = t < nt && v0 + x < V ? a.v[(size_t)(t0 + t) * a.ld + (size_t)h * V + v0 + x] : 0.f;
    }
    float sc[4][4], in[4][4], nq[4];
#pragma unroll
    for (int r = 0; r < 4; ++r) {
        nq[r] = 0.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) sc[r][e] = in[r][e] = 0.f;
    }
    const float* S = w.S + ((size_t)c * a.H + h) * D * V;
    const float* N = w.N + ((size_t)c * a.H + h) * D;
    for (int d0 = 0; d0 < D; d0 += DS) {
        __syncthreads();
        // a warp stages 8 state rows x 4 tokens at a time: whole sectors in, 32 different banks out
        {
            const int dl = tid & 7, tl = (tid >> 3) & 3, grp = tid >> 5;
#pragma unroll 4
            for (int u = grp; u < (DS / 8) * (CK / 4); u += 8) {
                const int d = (u % (DS / 8)) * 8 + dl, t = (u / (DS / 8)) * 4 + tl;
                const bool ok = t < nt && d0 + d < D;
                const size_t o = (size_t)(t0 + t) * a.ld + (size_t)h * D + d0 + d;
                qT[d * QP + t] = ok ? a.q[o] * a.q_scale : 0.f;
                kT[d * QP + t] = ok ? a.k[o] : 0.f;
            }
        }
#pragma unroll 4
        for (int idx = tid; idx < DS * CT; idx += 256) {
            const int d = idx / CT, x = idx % CT;
            Ss[idx] = d0 + d < D && v0 + x < V ? S[(size_t)(d0 + d) * V + v0 + x] : 0.f;
        }
        if (tid < DS) nsl[tid] = d0 + tid < D ? N[d0 + tid] : 0.f;
        __syncthreads();
#pragma unroll 8
        for (int d = 0; d < DS; ++d) {
            const float4 q4 = *reinterpret_cast<const float4*>(qT + d * QP + 4 * ty), k4 = *reinterpret_cast<const float4*>(kT + d * QP + 4 * tx);
            const float4 sv = s4[d * (CT / 4) + tx];
            const float n = nsl[d];
            const float qr[4] = {q4.x, q4.y, q4.z, q4.w}, ke[4] = {k4.x, k4.y, k4.z, k4.w}, se[4] = {sv.x, sv.y, sv.z, sv.w};
#pragma unroll
            for (int r = 0; r < 4; ++r) {
                nq[r] = fmaf(qr[r], n, nq[r]);
#pragma unroll
                for (int e = 0; e < 4; ++e) {
                    sc[r][e] = fmaf(qr[r], ke[e], sc[r][e]);
                    in[r][e] = fmaf(qr[r], se[e], in[r][e]);
                }
            }
        }
    }
    __syncthreads();
    float den[4];
#pragma unroll
    for (int r = 0; r < 4; ++r) {
        const int t = 4 * ty + r;
        float sum = 0.f;
        const double ft = t < nt ? Fs[t + 1] - (double)ms[t + 1] : 0.0;
#pragma unroll
        for (int e = 0; e < 4; ++e) {
            const int s = 4 * tx + e;
            const float wt = t < nt && s <= t ? expf((float)(ft - Fs[s + 1] + (double)is[s])) : 0.f;
            sc[r][e] *= wt;
            sum += sc[r][e];
        }
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) sum += __shfl_xor_sync(0xffffffffu, sum, o);
        const float g = t < nt ? expf((float)(ft - Fs[0] + (double)ms[0])) : 0.f;
        den[r] = t < nt ? fmaxf(fabsf(fmaf(g, nq[r], sum)), expf(-ms[t + 1])) + a.den_eps : 1.f;
#pragma unroll
        for (int e = 0; e < 4; ++e) in[r][e] *= g;
    }
#pragma unroll
    for (int e = 0; e < 4; ++e)
        *reinterpret_cast<float4*>(pT + (4 * tx + e) * QP + 4 * ty) = make_float4(sc[0][e], sc[1][e], sc[2][e], sc[3][e]);
    __syncthreads();
#pragma unroll 8
    for (int s = 0; s < CK; ++s) {
        const float4 p4 = *reinterpret_cast<const float4*>(pT + s * QP + 4 * ty), vv = v4[s * (CT / 4) + tx];
        const float pr[4] = {p4.x, p4.y, p4.z, p4.w}, ve[4] = {vv.x, vv.y, vv.z, vv.w};
#pragma unroll
        for (int r = 0; r < 4; ++r)
#pragma unroll
            for (int e = 0; e < 4; ++e) in[r][e] = fmaf(pr[r], ve[e], in[r][e]);
    }
#pragma unroll
    for (int r = 0; r < 4; ++r) {
        const int t = 4 * ty + r;
        if (t >= nt) continue;
        float* o = a.o + ((size_t)(t0 + t) * a.H + h) * V + v0 + 4 * tx;
        const float inv = 1.0f / den[r];
        if (V % 4 == 0 && v0 + 4 * tx < V) {
            *reinterpret_cast<float4*>(o) = make_float4(in[r][0] * inv, in[r][1] * inv, in[r][2] * inv, in[r][3] * inv);
        } else {
#pragma unroll
            for (int e = 0; e < 4; ++e)
                if (v0 + 4 * tx + e < V) o[e] = in[r][e] * inv;
        }
    }
}

// ------------------------------------------------------------------------------------------------ host side
template <int CH>
static int launch_scan(const CcSeqMlstm* a, cudaStream_t st) {
    const int P = (a->D + CH - 1) / CH, TB = a->T < SCAN_TB ? a->T : SCAN_TB;
    const size_t smem = sizeof(float) * (size_t)TB * (2 * P * CH + SCAN_J + P * SCAN_J);
    static size_t configured = 40 * 1024;      // beside the static arrays
    if (smem > configured) {
        configured = smem;
        if (cudaFuncSetAttribute(mlstm_scan_kernel<CH>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem) != cudaSuccess)
            return cuda_check("mlstm: shared memory");
    }
    mlstm_scan_kernel<CH><<<dim3(a->H, (a->V + SCAN_J - 1) / SCAN_J), (P + 1) * 32, smem, st>>>(*a);
    return cuda_check("mlstm_scan_kernel");
}

constexpr int SCAN_MAX_D = 32 * SCAN_ND, CHUNKS_FROM = 32;

static bool by_scan(int T, int D, int path) {
    return path == CC_MLSTM_SCAN || (path == CC_MLSTM_AUTO && T < CHUNKS_FROM && D <= SCAN_MAX_D);
}

static int check_bounded(const CcSeqBounded& b) { return b.w == nullptr || (b.alpha != nullptr && b.b != nullptr); }

static uintptr_t addr(const CcSeqBounded& b) { return (uintptr_t)b.w | (uintptr_t)b.b; }

}  // namespace ccc

using namespace ccc;

extern "C" {

int cc_seq_bounded_sum(const CcSeqBoundedSum* a, void* stream) {
    if (!a || !a->x || a->T < 1 || a->E < 1 || (!a->x_out && !a->h) || (a->y && !a->out_norm.w) || (a->h && !a->next_norm.w) ||
        !check_bounded(a->out_norm) || !check_bounded(a->next_norm) || (a->rows && a->x_out == a->x))
        return fail(CC_SEQ_ERR_INVALID_ARG, "bounded_sum: bad argument");
    if (a->act_dtype != CC_DT_F32 && a->act_dtype != CC_DT_BF16) return fail(CC_SEQ_ERR_INVALID_ARG, "unknown element type");
    cudaStream_t st = (cudaStream_t)stream;
    const uintptr_t all = (uintptr_t)a->x | (uintptr_t)a->y | (uintptr_t)a->add | (uintptr_t)a->x_out | (uintptr_t)a->h | addr(a->out_norm) | addr(a->next_norm);
    // one row: a thread per channel spreads it over more of the GPU
    const bool vec = a->T > 1 && a->E % 4 == 0 && a->ldy % 4 == 0 && (all & 15) == 0;
    const dim3 grid = row_grid(a->T, a->E, vec ? 4 : 1);
    if (a->act_dtype == CC_DT_BF16) {
        if (vec) bounded_sum_kernel<bf16, 4><<<grid, 128, 0, st>>>(*a);
        else bounded_sum_kernel<bf16, 1><<<grid, 128, 0, st>>>(*a);
    } else {
        if (vec) bounded_sum_kernel<float, 4><<<grid, 128, 0, st>>>(*a);
        else bounded_sum_kernel<float, 1><<<grid, 128, 0, st>>>(*a);
    }
    return cuda_check("bounded_sum_kernel");
}

int cc_seq_embed_bounded(const int32_t* tokens, const void* embed, int32_t table_dtype, const CcSeqBounded* emb, float* x,
                         const CcSeqBounded* next, void* h, int32_t act_dtype, int32_t T, int32_t E, void* stream) {
    if (!tokens || !embed || !emb || !emb->w || !x || T < 1 || E < 1 || (h && (!next || !next->w)) || !check_bounded(*emb) ||
        (next && !check_bounded(*next)))
        return fail(CC_SEQ_ERR_INVALID_ARG, "embed_bounded: bad argument");
    cudaStream_t st = (cudaStream_t)stream;
    CcSeqBounded nx = {nullptr, nullptr, nullptr};
    if (next) nx = *next;
    const uintptr_t all = (uintptr_t)embed | (uintptr_t)x | (uintptr_t)h | addr(*emb) | addr(nx);
    const bool vec = T > 1 && E % 4 == 0 && (all & 15) == 0;
    const dim3 grid = row_grid(T, E, vec ? 4 : 1);
#define EB(ST, AT)                                                                                                        \
    {                                                                                                                     \
        if (vec) embed_bounded_kernel<ST, AT, 4><<<grid, 128, 0, st>>>(tokens, (const ST*)embed, *emb, x, nx, (AT*)h, T, E); \
        else embed_bounded_kernel<ST, AT, 1><<<grid, 128, 0, st>>>(tokens, (const ST*)embed, *emb, x, nx, (AT*)h, T, E);     \
    }
    if (table_dtype == CC_DT_BF16 && act_dtype == CC_DT_BF16) EB(bf16, bf16)
    else if (table_dtype == CC_DT_BF16 && act_dtype == CC_DT_F32) EB(bf16, float)
    else if (table_dtype == CC_DT_F32 && act_dtype == CC_DT_F32) EB(float, float)
    else if (table_dtype == CC_DT_F32 && act_dtype == CC_DT_BF16) EB(float, bf16)
    else return fail(CC_SEQ_ERR_INVALID_ARG, "unknown element type");
#undef EB
    return cuda_check("embed_bounded_kernel");
}

uint64_t cc_seq_mlstm_workspace(int32_t T, int32_t H, int32_t D, int32_t V, int32_t path) {
    return by_scan(T, D, path) ? 0 : chunk_space(nullptr, nullptr, T, H, D, V);
}

int cc_seq_mlstm(const CcSeqMlstm* a, void* stream) {
    if (!a || !a->q || !a->k || !a->v || !a->i_raw || !a->f_raw || !a->i_bias || !a->f_bias || !a->state || !a->aux || !a->o ||
        a->T < 1 || a->H < 1 || a->D < 1 || a->V < 1 || !(a->gate_cap > 0.f) || a->path < CC_MLSTM_AUTO || a->path > CC_MLSTM_CHUNKS)
        return fail(CC_SEQ_ERR_INVALID_ARG, "mlstm: bad argument");
    cudaStream_t st = (cudaStream_t)stream;
    if (by_scan(a->T, a->D, a->path)) {
        if (a->D > SCAN_MAX_D) return fail(CC_SEQ_ERR_UNSUPPORTED_SHAPE, "mlstm: the scan holds up to 512 state rows per head");
        if (a->D <= 128) return launch_scan<8>(a, st);
        if (a->D <= 256) return launch_scan<16>(a, st);
        return launch_scan<32>(a, st);
    }
    if (!a->workspace || ((uintptr_t)a->workspace & 15) || a->workspace_bytes < chunk_space(nullptr, nullptr, a->T, a->H, a->D, a->V))
        return fail(CC_SEQ_ERR_INVALID_ARG, "mlstm: workspace missing, unaligned or too small");
    const int td = (a->D + CT - 1) / CT, tv = (a->V + CT - 1) / CT;
    if (a->H > 65535 || td * tv > 65535) return fail(CC_SEQ_ERR_UNSUPPORTED_SHAPE, "mlstm: too many heads or tiles");
    ChunkSpace w;
    chunk_space(&w, a->workspace, a->T, a->H, a->D, a->V);
    mlstm_gates_kernel<<<a->H, GATE_THREADS, 0, st>>>(*a, w);
    mlstm_chunk_sums_kernel<<<dim3(w.chunks, a->H, td * tv), 256, 0, st>>>(*a, w);
    mlstm_pass_kernel<<<dim3((unsigned)(((size_t)a->D * a->V + a->D + 255) / 256), a->H), 256, 0, st>>>(*a, w);
    mlstm_chunk_out_kernel<<<dim3(w.chunks, a->H, tv), 256, 0, st>>>(*a, w);
    return cuda_check("mlstm chunk kernels");
}

}  // extern "C"
