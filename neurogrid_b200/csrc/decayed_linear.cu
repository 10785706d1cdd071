// Linear attention whose state decays by one number per head and token, over a ragged batch; two forms:
//
//   lightning:  q, k, v <- silu(.) of the projections;  S_t = lambda_h S_(t-1) + k_t v_t^T;  o_t = S_t^T q_t
//   mLSTM:      i_t = c tanh((x_i + b_i) / c), f_t = log sigmoid(c tanh((x_f + b_f) / c))      (c: the gates' soft cap)
//               m_t = max(f_t + m_(t-1), i_t), m before the first token 0
//               S_t = exp(f_t + m_(t-1) - m_t) S_(t-1) + exp(i_t - m_t) k_t v_t^T,   n_t likewise with k_t alone
//               o_t = s S_t^T q_t / (max(|s n_t . q_t|, exp(-m_t)) + 1e-6),  s = dk^(-1/2)
//   both:       out = o over its root mean square (over a head, or over all heads together) * w * sigmoid(gate) * scale
//
// Input rows are [q (nH*dk) | k (nH*dk) | v (nH*dv) | gate (nH*dv)] of the activation type; the gates' preactivations
// [i (nH) | f (nH)] of the mLSTM are float32.  silu is rounded to the activation type (it belongs to the projection);
// everything behind that is float32: gates, decays, stabiliser, state, sums, norm, output gate.
// State per request: S [nH, dk, dv]; the mLSTM also (n [dk], m) per head, once for every slice of DL_SLICE value
// columns (blocks that take different slices of a head share nothing, so each keeps a copy that it alone reads and
// writes in the token-by-token kernel).
//
// Token by token (any head sizes, both activation types): a block per (entry, head, slice of value columns) walks the
// entry's tokens in order; a warp keeps 16 rows of the slice's columns in registers, a lane per column.  Tokens are
// staged eight at a time and the warps' partial sums of the eight are added at once.  A token's arithmetic does not
// depend on how its request was cut or on what else is in the step.
//
// Chunk by chunk (bfloat16, long portions, head sizes in sixteens): chunks of DC tokens side by side on the tensor cores.
// With S, n, m the state before a chunk, F_t the sum of the log decays of its tokens up to t (a power of lambda for
// lightning) and N its last token:
//     w(t, s) = exp(F_t - F_s + i_s - m_t)                    (lightning: lambda^(t - s))
//     U       = sum_s w(N, s) k_s v_s^T                       what the chunk adds;   S' = exp(F_N + m - m_N) S + U
//     o_t     = sum_(s <= t) (q_t . k_s) w(t, s) v_s + exp(F_t + m - m_t) S^T q_t     (numerator; the denominator's
//               n_t . q_t is the same sum without v)
// and m_t = max(m + F_t, max_(s <= t) (F_t - F_s + i_s)), so every exponent is at most 0.  `gates` forms F, i, m of all
// tokens (a max-plus scan), `local` U of every chunk, `scan` walks a request's chunks and leaves each chunk's S where its
// U was, `out` forms o, `finish` norms and gates.  q, k, v are bfloat16, so q . k is a float32 sum of exact products; the
// float32 operands (weighted scores, weighted keys, the state) enter the tensor cores as three bfloat16 terms
// hi + mid + lo (what is left is below 2^-24 of the value), accumulated in float32.  The two routes differ by rounding.
// Chunk c of entry e uses slot cu_q[e] / DC + e + c of the scratch: slots of different entries do not meet, and
// rows / DC + entries + 1 slots are enough.
#include "ng_common.cuh"

typedef __nv_bfloat16 bf16;

#define DL_SLICE 32        // value columns of a block of the token-by-token kernel
#define DL_ROWS 16         // rows of S a warp keeps
#define DL_TOKENS 8        // tokens staged at a time
#define DL_MAX_WARPS 32    // dk <= 512
#define DC 64              // tokens of a chunk
#define DC_THREADS 128

enum { DL_LIGHTNING = 0, DL_MLSTM = 1 };

struct DlGeom {
    int nH, dk, dv;
    int g_parts;               // mLSTM: float32 partial sums the gates' preactivations come as (1: whole)
    size_t g_stride;           // ... elements between them
};

__device__ __forceinline__ float dl_silu(float z) { return z / (1.f + expf(-z)); }
// silu as the activation type holds it: what a projection with its activation would store (bfloat16: through the fast
// exponential and division, whose errors are far below that rounding)
__device__ __forceinline__ float dl_silu_fast(float z) { return __fdividef(z, 1.f + __expf(-z)); }
template <typename T>
__device__ __forceinline__ float dl_silu_as(float z) {
    if (sizeof(T) == 4) return dl_silu(z);
    T r;
    ng_st(&r, dl_silu_fast(z));
    return ng_ld(&r);
}
__device__ __forceinline__ float dl_log_sigmoid(float z) { return fminf(z, 0.f) - log1pf(expf(-fabsf(z))); }
// the log gates of one row and head; `gr`: the row's preactivations i | f, or n_part partial sums of them, `stride` apart
__device__ __forceinline__ void dl_log_gates(const float* gr, int head, int nH, int n_part, size_t stride, float bi, float bf,
                                             float cap, float& li, float& lf) {
    float xi = 0.f, xf = 0.f;
#pragma unroll 4
    for (int s = 0; s < n_part; ++s) {
        xi += gr[s * stride + head];
        xf += gr[s * stride + nH + head];
    }
    li = cap * tanhf((xi + bi) / cap);
    lf = dl_log_sigmoid(cap * tanhf((xf + bf) / cap));
}

// -------------------------------------------------------------------------------------------- token by token
template <typename T, int MODE>
__global__ void __launch_bounds__(32 * DL_MAX_WARPS)
dl_step_kernel(const T* __restrict__ x, const float* __restrict__ gates, const float* __restrict__ gate_bias,
               const float* __restrict__ decay, float cap, float* __restrict__ state, float* __restrict__ nm_state,
               float* __restrict__ o_raw, const int* __restrict__ cu_q, const int* __restrict__ ctx_before,
               const int* __restrict__ slots, DlGeom geo) {
    extern __shared__ float sm[];
    const int dk = geo.dk, dv = geo.dv, nH = geo.nH;
    const int G = blockDim.x >> 5;
    float* qs = sm;                                    // [DL_TOKENS][dk]
    float* ks = qs + DL_TOKENS * dk;                   // [DL_TOKENS][dk]
    float* vs = ks + DL_TOKENS * dk;                   // [DL_TOKENS][32]
    float* part = vs + DL_TOKENS * 32;                 // [DL_TOKENS][G][32]
    float* npart = part + DL_TOKENS * G * 32;          // [DL_TOKENS][G]
    __shared__ float keep_s[DL_TOKENS], add_s[DL_TOKENS], em_s[DL_TOKENS];
    ng_pdl_trigger();
    const int e = blockIdx.x, head = blockIdx.y, slice = blockIdx.z, slices = gridDim.z;
    const int tid = threadIdx.x, lane = tid & 31, g = tid >> 5;
    const int q0 = cu_q[e], qlen = cu_q[e + 1] - q0;
    const int col = slice * DL_SLICE + lane;
    const bool live = col < dv;
    const int i0 = g * DL_ROWS;
    float s[DL_ROWS];
    float nreg = 0.f, m = 0.f;
    float* S = nullptr;
    float* nm = nullptr;
    if (qlen > 0) {                                    // what earlier steps left: read before the wait
        S = state + ((size_t)slots[e] * nH + head) * dk * dv;
        const bool has = ctx_before[e] > 0;
#pragma unroll
        for (int r = 0; r < DL_ROWS; ++r)
            s[r] = (has && live && i0 + r < dk) ? S[(size_t)(i0 + r) * dv + col] : 0.f;
        if (MODE == DL_MLSTM) {
            nm = nm_state + (((size_t)slots[e] * nH + head) * slices + slice) * (dk + 1);
            if (has) {
                if (tid < dk) nreg = nm[tid];
                m = nm[dk];
            }
        }
    }
    ng_pdl_wait();
    if (qlen <= 0) return;
    x = ng_after_wait(x);
    const float* gt = ng_after_wait(gates);
    const size_t ld = 2 * (size_t)nH * (dk + dv);
    const size_t off_q = (size_t)head * dk, off_k = (size_t)nH * dk + off_q, off_v = 2 * (size_t)nH * dk + (size_t)head * dv;
    const float lam = MODE == DL_LIGHTNING ? decay[head * (DC + 1) + 1] : 0.f;
    const float qscale = MODE == DL_MLSTM ? rsqrtf((float)dk) : 1.f;
    for (int t0 = 0; t0 < qlen; t0 += DL_TOKENS) {
        const int nt = min(DL_TOKENS, qlen - t0);
        for (int idx = tid; idx < nt * dk; idx += blockDim.x) {
            const int t = idx / dk, i = idx - t * dk;
            const T* row = x + (size_t)(q0 + t0 + t) * ld;
            float qv = ng_ld(row + off_q + i), kv = ng_ld(row + off_k + i);
            if (MODE == DL_LIGHTNING) { qv = dl_silu_as<T>(qv); kv = dl_silu_as<T>(kv); }
            qs[t * dk + i] = qv * qscale;
            ks[t * dk + i] = kv;
        }
        for (int idx = tid; idx < nt * 32; idx += blockDim.x) {
            const int c = slice * DL_SLICE + (idx & 31);
            float v = c < dv ? ng_ld(x + (size_t)(q0 + t0 + (idx >> 5)) * ld + off_v + c) : 0.f;
            if (MODE == DL_LIGHTNING) v = dl_silu_as<T>(v);
            vs[idx] = v;
        }
        if (MODE == DL_MLSTM && g == 0) {              // a lane per token forms its gates; the maximum runs through the lanes
            float li = 0.f, lf = 0.f;
            if (lane < nt) {
                const float* gr = gt + (size_t)(q0 + t0 + lane) * 2 * nH;
                dl_log_gates(gr, head, nH, geo.g_parts, geo.g_stride, gate_bias[head], gate_bias[nH + head], cap, li, lf);
            }
            float mm = m, keep = 0.f, add = 0.f, em = 0.f;
            for (int t = 0; t < nt; ++t) {
                const float ft = __shfl_sync(0xffffffffu, lf, t), it = __shfl_sync(0xffffffffu, li, t);
                const float nx = fmaxf(ft + mm, it);
                if (lane == t) { keep = ft + mm - nx; add = it - nx; em = -nx; }
                mm = nx;
            }
            m = mm;
            if (lane < nt) { keep_s[lane] = expf(keep); add_s[lane] = expf(add); em_s[lane] = expf(em); }
        }
        __syncthreads();
        for (int t = 0; t < nt; ++t) {
            float kp = lam, vv = vs[t * 32 + lane];
            if (MODE == DL_MLSTM) { kp = keep_s[t]; vv *= add_s[t]; }
            float acc = 0.f;
            const float *qt = qs + t * dk + i0, *kt = ks + t * dk + i0;
#pragma unroll
            for (int r = 0; r < DL_ROWS; ++r)
                if (i0 + r < dk) {
                    s[r] = fmaf(kp, s[r], kt[r] * vv);
                    acc = fmaf(s[r], qt[r], acc);
                }
            part[(t * G + g) * 32 + lane] = acc;
            if (MODE == DL_MLSTM) {
                float nq = 0.f;
                if (tid < dk) {
                    nreg = fmaf(kp, nreg, add_s[t] * ks[t * dk + tid]);
                    nq = nreg * qs[t * dk + tid];
                }
                nq = ng_warp_sum(nq);
                if (lane == 0) npart[t * G + g] = nq;
            }
        }
        __syncthreads();
        for (int idx = tid; idx < nt * 32; idx += blockDim.x) {
            const int t = idx >> 5, c = slice * DL_SLICE + (idx & 31);
            if (c >= dv) continue;
            float o = 0.f;
            for (int gg = 0; gg < G; ++gg) o += part[(t * G + gg) * 32 + (idx & 31)];
            if (MODE == DL_MLSTM) {
                float den = 0.f;
                for (int gg = 0; gg < G; ++gg) den += npart[t * G + gg];
                o /= fmaxf(fabsf(den), em_s[t]) + 1e-6f;
            }
            o_raw[(size_t)(q0 + t0 + t) * nH * dv + (size_t)head * dv + c] = o;
        }
        __syncthreads();
    }
    if (live) {
#pragma unroll
        for (int r = 0; r < DL_ROWS; ++r)
            if (i0 + r < dk) S[(size_t)(i0 + r) * dv + col] = s[r];
    }
    if (MODE == DL_MLSTM) {
        if (tid < dk) nm[tid] = nreg;
        if (tid == 0) nm[dk] = m;
    }
}

// -------------------------------------------------------------------------------------------- head norm and output gate
// out[row, c] = o[row, c] / sqrt(mean over the c's group of o^2 + eps) * w[c] * sigmoid(gate[row, c]) * scale; groups of
// `group` neighbouring columns (a head, or the whole row).  A block per row; columns dealt to warps group by group, or,
// when the row is one group, to the whole block.  Rows of `out` lie ldo elements apart, rows of `gate` ldg.
template <typename T>
__global__ void __launch_bounds__(256)
dl_finish_kernel(const float* __restrict__ o, const T* __restrict__ gate, const float* __restrict__ w, T* __restrict__ out,
                 const int* __restrict__ row_entry, int width, int group, int ldg, int ldo, float eps, float scale) {
    __shared__ float red[32];
    ng_pdl_trigger();
    ng_pdl_wait();
    const size_t row = blockIdx.x;
    T* orow = out + row * (size_t)ldo;
    if (row_entry[row] < 0) {                          // padding row: defined output
        for (int c = threadIdx.x; c < width; c += blockDim.x) ng_st(orow + c, 0.f);
        return;
    }
    const float* in = o + row * (size_t)width;
    const T* gr = gate + row * (size_t)ldg;
    if (group == width) {
        float ss = 0.f;
        for (int c = threadIdx.x; c < width; c += blockDim.x) ss = fmaf(in[c], in[c], ss);
        const float r = rsqrtf(ng_block_sum(ss, red) / (float)width + eps);
        for (int c = threadIdx.x; c < width; c += blockDim.x)
            ng_st(orow + c, in[c] * r * w[c] * (scale / (1.f + expf(-ng_ld(gr + c)))));
        return;
    }
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, warps = blockDim.x >> 5;
    for (int h = warp; h < width / group; h += warps) {
        float ss = 0.f;
        for (int c = h * group + lane; c < (h + 1) * group; c += 32) ss = fmaf(in[c], in[c], ss);
        const float r = rsqrtf(ng_warp_sum(ss) / (float)group + eps);
        for (int c = h * group + lane; c < (h + 1) * group; c += 32)
            ng_st(orow + c, in[c] * r * w[c] * (scale / (1.f + expf(-ng_ld(gr + c)))));
    }
}

// The same in one pass over memory: four columns a thread and step, at most NV steps, all loads issued before the norm's
// sum.  A warp per (row, group), or (WHOLE) a block per row whose columns are one group.
__device__ __forceinline__ float4 dl_ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ float4 dl_ld4(const bf16* p) {
    const uint2 u = *reinterpret_cast<const uint2*>(p);
    return make_float4(__uint_as_float(u.x << 16), __uint_as_float(u.x & 0xffff0000u), __uint_as_float(u.y << 16),
                       __uint_as_float(u.y & 0xffff0000u));
}
__device__ __forceinline__ void dl_st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ void dl_st4(bf16* p, float4 v) {
    const __nv_bfloat162 a = __floats2bfloat162_rn(v.x, v.y), b = __floats2bfloat162_rn(v.z, v.w);
    *reinterpret_cast<uint2*>(p) = make_uint2(*reinterpret_cast<const uint32_t*>(&a), *reinterpret_cast<const uint32_t*>(&b));
}
template <typename T, bool WHOLE, int NV>
__global__ void __launch_bounds__(512)
dl_finish_vec_kernel(const float* __restrict__ o, const T* __restrict__ gate, const float* __restrict__ w, T* __restrict__ out,
                     const int* __restrict__ row_entry, int n_rows, int width, int group, int ldg, int ldo, float eps, float scale) {
    __shared__ float red[32];
    ng_pdl_trigger();
    const int groups = width / group;
    const size_t unit = WHOLE ? blockIdx.x : (size_t)blockIdx.x * (blockDim.x >> 5) + (threadIdx.x >> 5);
    const int me = WHOLE ? threadIdx.x : threadIdx.x & 31, step = 4 * (WHOLE ? blockDim.x : 32);
    const bool mine = unit < (size_t)n_rows * groups;
    const size_t row = mine ? unit / groups : 0;
    const int c0 = (int)(unit % groups) * group;
    float4 wv[NV];
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = 4 * me + k * step;
        wv[k] = mine && c < group ? dl_ld4(w + c0 + c) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    ng_pdl_wait();
    if (!mine) return;                                 // (WHOLE: never; else a whole warp)
    const float* in = ng_after_wait(o) + row * (size_t)width + c0;
    const T* gr = ng_after_wait(gate) + row * (size_t)ldg + c0;
    const bool real = row_entry[row] >= 0;             // padding row: zeros
    float4 v[NV], g[NV];
    float ss = 0.f;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = 4 * me + k * step;
        v[k] = g[k] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (real && c < group) { v[k] = dl_ld4(in + c); g[k] = dl_ld4(gr + c); }
    }
#pragma unroll
    for (int k = 0; k < NV; ++k) ss += v[k].x * v[k].x + v[k].y * v[k].y + v[k].z * v[k].z + v[k].w * v[k].w;
    ss = WHOLE ? ng_block_sum(ss, red) : ng_warp_sum(ss);
    const float r = rsqrtf(ss / (float)group + eps);
    T* orow = out + row * (size_t)ldo + c0;
#pragma unroll
    for (int k = 0; k < NV; ++k) {
        const int c = 4 * me + k * step;
        if (c < group)
            dl_st4(orow + c, make_float4(v[k].x * r * wv[k].x * (scale / (1.f + expf(-g[k].x))),
                                         v[k].y * r * wv[k].y * (scale / (1.f + expf(-g[k].y))),
                                         v[k].z * r * wv[k].z * (scale / (1.f + expf(-g[k].z))),
                                         v[k].w * r * wv[k].w * (scale / (1.f + expf(-g[k].w)))));
    }
}

// -------------------------------------------------------------------------------------------- chunk by chunk
__device__ __forceinline__ void dl_ldsm_x4(uint32_t (&r)[4], const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void dl_ldsm_x4_t(uint32_t (&r)[4], const void* p) {
    const uint32_t a = (uint32_t)__cvta_generic_to_shared(p);
    asm volatile("ldmatrix.sync.aligned.m8n8.x4.trans.shared.b16 {%0,%1,%2,%3}, [%4];"
                 : "=r"(r[0]), "=r"(r[1]), "=r"(r[2]), "=r"(r[3]) : "r"(a));
}
__device__ __forceinline__ void dl_mma(float (&c)[4], const uint32_t (&a)[4], uint32_t b0, uint32_t b1) {
    asm volatile("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0,%1,%2,%3}, {%4,%5,%6,%7}, {%8,%9}, {%0,%1,%2,%3};"
                 : "+f"(c[0]), "+f"(c[1]), "+f"(c[2]), "+f"(c[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b0), "r"(b1));
}
__device__ __forceinline__ uint32_t dl_pack(float x, float y) {
    const __nv_bfloat162 h = __floats2bfloat162_rn(x, y);
    return *reinterpret_cast<const uint32_t*>(&h);
}
// a pair of float32 values as bfloat16 terms hi + mid + lo
__device__ __forceinline__ void dl_split3(float x, float y, uint32_t& hi, uint32_t& mid, uint32_t& lo) {
    hi = dl_pack(x, y);
    const float xr = x - __uint_as_float(hi << 16), yr = y - __uint_as_float(hi & 0xffff0000u);
    mid = dl_pack(xr, yr);
    lo = dl_pack(xr - __uint_as_float(mid << 16), yr - __uint_as_float(mid & 0xffff0000u));
}

// acc[16 x N] += (hi + mid + lo)[16 x 16] v[16 x N], v in shared memory (`v`: this lane's row and column of the first
// group of 16 columns); smallest terms first, the column groups taking turns so that an accumulator's products are apart
template <int N>
__device__ __forceinline__ void dl_add_split(float (&acc)[N / 8][4], const uint32_t (&hi)[4], const uint32_t (&mid)[4],
                                             const uint32_t (&lo)[4], const bf16* v) {
    uint32_t b[N / 16][4];
#pragma unroll
    for (int x = 0; x < N / 16; ++x) dl_ldsm_x4_t(b[x], v + x * 16);
#pragma unroll
    for (int term = 0; term < 3; ++term) {
        const uint32_t (&a)[4] = term == 0 ? lo : term == 1 ? mid : hi;
#pragma unroll
        for (int x = 0; x < N / 16; ++x) {
            dl_mma(acc[2 * x], a, b[x][0], b[x][1]);
            dl_mma(acc[2 * x + 1], a, b[x][2], b[x][3]);
        }
    }
}

// columns [c0, c0 + cols) of n rows (64 at most; the rest zero) into shared memory, 16 bytes at a time, silu applied
// for lightning; dst row pitch `pitch` elements
template <int MODE>
__device__ __forceinline__ void dl_load_tile(bf16* dst, int pitch, const bf16* __restrict__ src, size_t ld, int cols, int n) {
    const int per = cols / 8;
    for (int idx = threadIdx.x; idx < DC * per; idx += DC_THREADS) {
        const int t = idx / per, c = (idx - t * per) * 8;
        uint4 v = make_uint4(0u, 0u, 0u, 0u);
        if (t < n) {
            v = *reinterpret_cast<const uint4*>(src + (size_t)t * ld + c);
            if (MODE == DL_LIGHTNING) {
                uint32_t* u = reinterpret_cast<uint32_t*>(&v);
#pragma unroll
                for (int k = 0; k < 4; ++k)
                    u[k] = dl_pack(dl_silu_fast(__uint_as_float(u[k] << 16)), dl_silu_fast(__uint_as_float(u[k] & 0xffff0000u)));
            }
        }
        *reinterpret_cast<uint4*>(dst + t * pitch + c) = v;
    }
}

// mLSTM: per token a_t = F_t - m_t, b_t = F_t - i_t, exp(-m_t) -> tok [rows][nH] float4; per chunk its maximum before the
// first token and exp(F_N + m - m_N) -> chk [slots][nH] float2; the last maximum to the request's slot (every slice's
// copy).  A block per (entry, head): a warp per chunk (two tokens a lane), 32 chunks a round.
__global__ void __launch_bounds__(1024)
dl_gates_kernel(const float* __restrict__ gates, const float* __restrict__ gate_bias, float cap, float4* __restrict__ tok,
                float2* __restrict__ chk, float* __restrict__ nm_state, const int* __restrict__ cu_q,
                const int* __restrict__ ctx_before, const int* __restrict__ slots, DlGeom geo, int slices) {
    const int nH = geo.nH, dk = geo.dk;
    __shared__ float sum_s[32], top_s[32], m_s[33];
    ng_pdl_trigger();
    ng_pdl_wait();
    const int e = blockIdx.x, head = blockIdx.y;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int q0 = cu_q[e], qlen = cu_q[e + 1] - q0;
    if (qlen <= 0) return;
    float* nm = nm_state + ((size_t)slots[e] * nH + head) * slices * (dk + 1) + dk;
    const float bi = gate_bias[head], bf = gate_bias[nH + head];
    float m0 = ctx_before[e] > 0 ? *nm : 0.f;
    const int nc = (qlen + DC - 1) / DC;
    for (int c0 = 0; c0 < nc; c0 += 32) {
        const int c = c0 + warp, tb = c * DC + 2 * lane;
        float li[2], lf[2];
#pragma unroll
        for (int u = 0; u < 2; ++u) {
            li[u] = -INFINITY;                         // a token that is not there adds nothing and forgets nothing
            lf[u] = 0.f;
            if (tb + u < qlen) {
                const float* gr = gates + (size_t)(q0 + tb + u) * 2 * nH;
                dl_log_gates(gr, head, nH, geo.g_parts, geo.g_stride, bi, bf, cap, li[u], lf[u]);
            }
        }
        // F of the lane's two tokens: a scan of the pairs' sums
        float incl = lf[0] + lf[1];
#pragma unroll
        for (int d = 1; d < 32; d <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, incl, d);
            if (lane >= d) incl += up;
        }
        float prev = __shfl_up_sync(0xffffffffu, incl, 1);
        if (lane == 0) prev = 0.f;
        const float F0 = prev + lf[0], F1 = F0 + lf[1];
        // running maximum of i_s - F_s
        const float g0 = li[0] - F0, g1 = fmaxf(g0, li[1] - F1);
        float mx = g1;
#pragma unroll
        for (int d = 1; d < 32; d <<= 1) {
            const float up = __shfl_up_sync(0xffffffffu, mx, d);
            if (lane >= d) mx = fmaxf(mx, up);
        }
        float pm = __shfl_up_sync(0xffffffffu, mx, 1);
        if (lane == 0) pm = -INFINITY;
        const float Fn = __shfl_sync(0xffffffffu, F1, 31);             // (tokens that are not there have f = 0)
        const float top = __shfl_sync(0xffffffffu, mx, 31);
        if (lane == 0) { sum_s[warp] = Fn; top_s[warp] = top; }
        __syncthreads();
        if (threadIdx.x == 0) {
            float m = m0;
            for (int k = 0; k < 32; ++k) {
                m_s[k] = m;
                if (c0 + k < nc) m = sum_s[k] + fmaxf(m, top_s[k]);
            }
            m_s[32] = m;
        }
        __syncthreads();
        const float m_in = m_s[warp];
        m0 = m_s[32];
        if (c < nc) {
            const float mt0 = F0 + fmaxf(m_in, fmaxf(pm, g0)), mt1 = F1 + fmaxf(m_in, fmaxf(pm, g1));
            if (tb < qlen) tok[(size_t)(q0 + tb) * nH + head] = make_float4(F0 - mt0, F0 - li[0], expf(-mt0), 0.f);
            if (tb + 1 < qlen) tok[(size_t)(q0 + tb + 1) * nH + head] = make_float4(F1 - mt1, F1 - li[1], expf(-mt1), 0.f);
            if (lane == 0) {
                const float mn = Fn + fmaxf(m_in, top);
                chk[(size_t)(q0 / DC + e + c) * nH + head] = make_float2(m_in, expf(Fn + m_in - mn));
            }
        }
        __syncthreads();
    }
    for (int k = threadIdx.x; k < slices; k += blockDim.x) nm[(size_t)k * (dk + 1)] = m0;
}

// U of a chunk for one head and slice of DVS value columns (and, slice 0 of the mLSTM, the same sum without v)
template <int MODE, int DVS>
__global__ void __launch_bounds__(DC_THREADS)
dl_local_kernel(const bf16* __restrict__ x, const float4* __restrict__ tok, const float* __restrict__ decay,
                float* __restrict__ u_scratch, float* __restrict__ un_scratch, const int* __restrict__ cu_q, DlGeom geo) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int dk = geo.dk, dv = geo.dv, nH = geo.nH, KP = dk + 8;
    constexpr int VP = DVS + 8;
    bf16* Ks = reinterpret_cast<bf16*>(smem_raw);      // [DC][KP]
    bf16* Vs = Ks + DC * KP;                           // [DC][VP]
    __shared__ float ws[DC];
    ng_pdl_trigger();
    ng_pdl_wait();
    const int c = blockIdx.x, e = blockIdx.y, slices = dv / DVS;
    const int head = blockIdx.z / slices, sl = blockIdx.z % slices;
    const int q0 = cu_q[e], qlen = cu_q[e + 1] - q0;
    if (c * DC >= qlen) return;
    const int n = min(DC, qlen - c * DC), row0 = q0 + c * DC;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const size_t ld = 2 * (size_t)nH * (dk + dv);
    const bf16* xr = x + (size_t)row0 * ld;
    dl_load_tile<MODE>(Ks, KP, xr + (size_t)nH * dk + (size_t)head * dk, ld, dk, n);
    dl_load_tile<MODE>(Vs, VP, xr + 2 * (size_t)nH * dk + (size_t)head * dv + sl * DVS, ld, DVS, n);
    if (MODE == DL_LIGHTNING) {
        if (tid < DC) ws[tid] = tid < n ? decay[head * (DC + 1) + n - 1 - tid] : 0.f;
    } else if (tid < DC) {
        const float a_last = tok[(size_t)(row0 + n - 1) * nH + head].x;
        ws[tid] = tid < n ? expf(a_last - tok[(size_t)(row0 + tid) * nH + head].y) : 0.f;
    }
    __syncthreads();
    const size_t slot = (size_t)(q0 / DC + e + c) * nH + head;
    float* U = u_scratch + slot * dk * dv + sl * DVS;
    const int gq = lane >> 2, tq = lane & 3;
    for (int m0 = warp * 16; m0 < dk; m0 += 64) {
        float acc[DVS / 8][4];
#pragma unroll
        for (int j = 0; j < DVS / 8; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll
        for (int kk = 0; kk < DC / 16; ++kk) {
            uint32_t a[4], ah[4], am[4], al[4];
            // K^T: rows of the fragment are key coordinates, columns tokens
            dl_ldsm_x4_t(a, Ks + (kk * 16 + (lane >> 4) * 8 + (lane & 7)) * KP + m0 + ((lane >> 3) & 1) * 8);
#pragma unroll
            for (int u = 0; u < 4; ++u) {
                const int t = kk * 16 + 2 * tq + (u >> 1) * 8;
                dl_split3(__uint_as_float(a[u] << 16) * ws[t], __uint_as_float(a[u] & 0xffff0000u) * ws[t + 1], ah[u], am[u], al[u]);
            }
            dl_add_split<DVS>(acc, ah, am, al, Vs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VP + (lane >> 4) * 8);
        }
#pragma unroll
        for (int j = 0; j < DVS / 8; ++j) {
            *reinterpret_cast<float2*>(U + (size_t)(m0 + gq) * dv + j * 8 + 2 * tq) = make_float2(acc[j][0], acc[j][1]);
            *reinterpret_cast<float2*>(U + (size_t)(m0 + gq + 8) * dv + j * 8 + 2 * tq) = make_float2(acc[j][2], acc[j][3]);
        }
    }
    if (MODE == DL_MLSTM && sl == 0)
        for (int i = tid; i < dk; i += DC_THREADS) {
            float a = 0.f;
            for (int t = 0; t < n; ++t) a = fmaf(__bfloat162float(Ks[t * KP + i]), ws[t], a);
            un_scratch[slot * dk + i] = a;
        }
}

// Four neighbouring state elements of a (request, head) a thread: S before each chunk replaces the chunk's U; the last S'
// is the slot's.  Behind the dk*dv elements of S the mLSTM's n.
template <int MODE>
__global__ void __launch_bounds__(256)
dl_scan_kernel(float* __restrict__ u_scratch, float* __restrict__ un_scratch, float* __restrict__ state,
               float* __restrict__ nm_state, const float* __restrict__ decay, const float2* __restrict__ chk,
               const int* __restrict__ cu_q, const int* __restrict__ ctx_before, const int* __restrict__ slots, DlGeom geo,
               int step_slices) {
    constexpr int AHEAD = 8;                           // chunks whose additions are in flight at once
    ng_pdl_trigger();
    ng_pdl_wait();
    const int e = blockIdx.y, head = blockIdx.z, nH = geo.nH, dk = geo.dk, dv = geo.dv;
    const int n_s = dk * dv, i = 4 * (blockIdx.x * 256 + threadIdx.x);
    const int q0 = cu_q[e], qlen = cu_q[e + 1] - q0;
    const bool is_n = MODE == DL_MLSTM && i >= n_s;
    if (qlen <= 0 || (is_n ? i - n_s >= dk : i >= n_s)) return;
    const size_t slot0 = (size_t)(q0 / DC + e) * nH + head;
    const size_t unit = is_n ? dk : n_s;               // floats of a (chunk, head)
    float* U0 = (is_n ? un_scratch + (i - n_s) : u_scratch + i) + slot0 * unit;
    const size_t stride = (size_t)nH * unit;
    float* own = nullptr;
    float4 s = make_float4(0.f, 0.f, 0.f, 0.f);
    const bool has = ctx_before[e] > 0;
    if (is_n) {
        own = nm_state + ((size_t)slots[e] * nH + head) * step_slices * (dk + 1) + (i - n_s);     // rows of dk + 1: no 16-byte accesses
        if (has) s = make_float4(own[0], own[1], own[2], own[3]);
    } else {
        own = state + ((size_t)slots[e] * nH + head) * n_s + i;
        if (has) s = *reinterpret_cast<const float4*>(own);
    }
    const int nc = (qlen + DC - 1) / DC;
    float full = 1.f, last = 1.f;
    if (MODE == DL_LIGHTNING) {
        full = decay[head * (DC + 1) + DC];
        last = decay[head * (DC + 1) + qlen - (nc - 1) * DC];
    }
    for (int c0 = 0; c0 < nc; c0 += AHEAD) {
        float4 u[AHEAD];
        float f[AHEAD];
#pragma unroll
        for (int k = 0; k < AHEAD; ++k) {
            const int c = c0 + k;
            if (c < nc) {
                u[k] = *reinterpret_cast<const float4*>(U0 + (size_t)c * stride);
                f[k] = MODE == DL_LIGHTNING ? (c == nc - 1 ? last : full) : chk[slot0 + (size_t)c * nH].y;
            }
        }
#pragma unroll
        for (int k = 0; k < AHEAD; ++k) {
            const int c = c0 + k;
            if (c < nc) {
                *reinterpret_cast<float4*>(U0 + (size_t)c * stride) = s;
                s.x = fmaf(s.x, f[k], u[k].x);
                s.y = fmaf(s.y, f[k], u[k].y);
                s.z = fmaf(s.z, f[k], u[k].z);
                s.w = fmaf(s.w, f[k], u[k].w);
            }
        }
    }
    if (is_n) {
        for (int k = 0; k < step_slices; ++k) {
            float* d = own + (size_t)k * (dk + 1);
            d[0] = s.x; d[1] = s.y; d[2] = s.z; d[3] = s.w;
        }
    } else {
        *reinterpret_cast<float4*>(own) = s;
    }
}

template <int DVS>
static size_t dl_out_smem(int dk) {
    return ((size_t)2 * DC * (dk + 8) + (size_t)DC * (DVS + 8) + (size_t)3 * dk * (DVS + 8)) * sizeof(bf16) + (size_t)dk * sizeof(float);
}
template <int DVS>
static size_t dl_local_smem(int dk) {
    return ((size_t)DC * (dk + 8) + (size_t)DC * (DVS + 8)) * sizeof(bf16);
}

// o of a chunk for one head and slice of DVS value columns: a warp per 16 rows
template <int MODE, int DVS>
__global__ void __launch_bounds__(DC_THREADS)
dl_out_kernel(const bf16* __restrict__ x, const float4* __restrict__ tok, const float2* __restrict__ chk,
              const float* __restrict__ decay, const float* __restrict__ u_scratch, const float* __restrict__ un_scratch,
              float* __restrict__ o_raw, const int* __restrict__ cu_q, DlGeom geo) {
    extern __shared__ __align__(16) unsigned char smem_raw[];
    const int dk = geo.dk, dv = geo.dv, nH = geo.nH, KP = dk + 8;
    constexpr int VP = DVS + 8;
    bf16* Qs = reinterpret_cast<bf16*>(smem_raw);      // [DC][KP]
    bf16* Ks = Qs + DC * KP;                           // [DC][KP]
    bf16* Vs = Ks + DC * KP;                           // [DC][VP]
    bf16* Sh = Vs + DC * VP;                           // [3][dk][VP]: the state's terms hi, mid, lo
    float* ns = reinterpret_cast<float*>(Sh + (size_t)3 * dk * VP);      // [dk]
    __shared__ float a_s[DC], b_s[DC], em_s[DC], ein_s[DC], nq_s[DC], pw[DC + 1];
    ng_pdl_trigger();
    ng_pdl_wait();
    const int c = blockIdx.x, e = blockIdx.y, slices = dv / DVS;
    const int head = blockIdx.z / slices, sl = blockIdx.z % slices;
    const int q0 = cu_q[e], qlen = cu_q[e + 1] - q0;
    if (c * DC >= qlen) return;
    const int n = min(DC, qlen - c * DC), row0 = q0 + c * DC;
    const int tid = threadIdx.x, lane = tid & 31, warp = tid >> 5;
    const size_t ld = 2 * (size_t)nH * (dk + dv);
    const bf16* xr = x + (size_t)row0 * ld;
    dl_load_tile<MODE>(Qs, KP, xr + (size_t)head * dk, ld, dk, n);
    dl_load_tile<MODE>(Ks, KP, xr + (size_t)nH * dk + (size_t)head * dk, ld, dk, n);
    dl_load_tile<MODE>(Vs, VP, xr + 2 * (size_t)nH * dk + (size_t)head * dv + sl * DVS, ld, DVS, n);
    const size_t slot = (size_t)(q0 / DC + e + c) * nH + head;
    const float* Sb = u_scratch + slot * dk * dv + sl * DVS;
    for (int idx = tid; idx < dk * (DVS / 4); idx += DC_THREADS) {
        const int d = idx / (DVS / 4), v4 = (idx % (DVS / 4)) * 4;
        const float4 f = *reinterpret_cast<const float4*>(Sb + (size_t)d * dv + v4);
        uint2 h, m, l;
        dl_split3(f.x, f.y, h.x, m.x, l.x);
        dl_split3(f.z, f.w, h.y, m.y, l.y);
        bf16* dst = Sh + (size_t)d * VP + v4;
        *reinterpret_cast<uint2*>(dst) = h;
        *reinterpret_cast<uint2*>(dst + (size_t)dk * VP) = m;
        *reinterpret_cast<uint2*>(dst + (size_t)2 * dk * VP) = l;
    }
    const float scale = MODE == DL_MLSTM ? rsqrtf((float)dk) : 1.f;
    if (MODE == DL_LIGHTNING) {
        if (tid <= DC) pw[tid] = decay[head * (DC + 1) + tid];
        if (tid < DC) ein_s[tid] = decay[head * (DC + 1) + tid + 1];
    } else {
        for (int i = tid; i < dk; i += DC_THREADS) ns[i] = un_scratch[slot * dk + i];
        if (tid < DC) {
            const float m_in = chk[slot].x;
            float4 g = make_float4(0.f, 0.f, 1.f, 0.f);
            if (tid < n) g = tok[(size_t)(row0 + tid) * nH + head];
            a_s[tid] = g.x;
            b_s[tid] = g.y;
            em_s[tid] = g.z;
            ein_s[tid] = expf(g.x + m_in) * scale;
        }
    }
    __syncthreads();
    if (MODE == DL_MLSTM) {                            // n before the chunk with every row's q: two threads a row
        const int t = tid >> 1, h = tid & 1, half = dk / 2;
        float a = 0.f;
        for (int i = h * half; i < (h + 1) * half; ++i) a = fmaf(__bfloat162float(Qs[t * KP + i]), ns[i], a);
        a += __shfl_xor_sync(0xffffffffu, a, 1);
        if (h == 0) nq_s[t] = a * ein_s[t];
        __syncthreads();
    }
    const int w0 = warp * 16;
    if (w0 >= n) return;
    const int gq = lane >> 2, tq = lane & 3;
    const int ta = w0 + gq, tb = ta + 8;               // this thread's two rows
    float s[DC / 8][4], o[DVS / 8][4];
#pragma unroll
    for (int j = 0; j < DC / 8; ++j) s[j][0] = s[j][1] = s[j][2] = s[j][3] = 0.f;
#pragma unroll
    for (int j = 0; j < DVS / 8; ++j) o[j][0] = o[j][1] = o[j][2] = o[j][3] = 0.f;
    for (int kk = 0; kk < dk / 16; ++kk) {
        uint32_t qf[4];
        dl_ldsm_x4(qf, Qs + (w0 + (lane & 7) + ((lane >> 3) & 1) * 8) * KP + kk * 16 + (lane >> 4) * 8);
#pragma unroll
        for (int jp = 0; jp < DC / 16; ++jp)
            if (jp <= warp) {                          // tokens behind the warp's rows are not seen
                uint32_t b[4];
                dl_ldsm_x4(b, Ks + (jp * 16 + (lane & 7) + (lane >> 4) * 8) * KP + kk * 16 + ((lane >> 3) & 1) * 8);
                dl_mma(s[2 * jp], qf, b[0], b[1]);
                dl_mma(s[2 * jp + 1], qf, b[2], b[3]);
            }
#pragma unroll
        for (int term = 2; term >= 0; --term) {        // smallest terms first
            const bf16* St = Sh + ((size_t)term * dk + kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VP + (lane >> 4) * 8;
#pragma unroll
            for (int np = 0; np < DVS / 16; ++np) {
                uint32_t b[4];
                dl_ldsm_x4_t(b, St + np * 16);
                dl_mma(o[2 * np], qf, b[0], b[1]);
                dl_mma(o[2 * np + 1], qf, b[2], b[3]);
            }
        }
    }
    const float ea = ein_s[ta], eb = ein_s[tb];
#pragma unroll
    for (int j = 0; j < DVS / 8; ++j) { o[j][0] *= ea; o[j][1] *= ea; o[j][2] *= eb; o[j][3] *= eb; }
    float den_a = 0.f, den_b = 0.f;
    const float aa = MODE == DL_MLSTM ? a_s[ta] : 0.f, ab = MODE == DL_MLSTM ? a_s[tb] : 0.f;
#pragma unroll
    for (int j = 0; j < DC / 8; ++j) {
        if (j / 2 > warp) break;
#pragma unroll
        for (int u = 0; u < 4; ++u) {
            const int ts = j * 8 + 2 * tq + (u & 1), t = u < 2 ? ta : tb;
            float w = 0.f;
            if (ts <= t) w = MODE == DL_LIGHTNING ? pw[t - ts] : expf((u < 2 ? aa : ab) - b_s[ts]) * scale;
            s[j][u] *= w;
            if (MODE == DL_MLSTM) { if (u < 2) den_a += s[j][u]; else den_b += s[j][u]; }
        }
    }
#pragma unroll
    for (int kk = 0; kk < DC / 16; ++kk) {
        if (kk > warp) break;
        uint32_t ah[4], am[4], al[4];
        dl_split3(s[2 * kk][0], s[2 * kk][1], ah[0], am[0], al[0]);
        dl_split3(s[2 * kk][2], s[2 * kk][3], ah[1], am[1], al[1]);
        dl_split3(s[2 * kk + 1][0], s[2 * kk + 1][1], ah[2], am[2], al[2]);
        dl_split3(s[2 * kk + 1][2], s[2 * kk + 1][3], ah[3], am[3], al[3]);
        dl_add_split<DVS>(o, ah, am, al, Vs + (kk * 16 + (lane & 7) + ((lane >> 3) & 1) * 8) * VP + (lane >> 4) * 8);
    }
    float ra = 1.f, rb = 1.f;
    if (MODE == DL_MLSTM) {
        den_a += __shfl_xor_sync(0xffffffffu, den_a, 1);
        den_a += __shfl_xor_sync(0xffffffffu, den_a, 2);
        den_b += __shfl_xor_sync(0xffffffffu, den_b, 1);
        den_b += __shfl_xor_sync(0xffffffffu, den_b, 2);
        ra = 1.f / (fmaxf(fabsf(den_a + nq_s[ta]), em_s[ta]) + 1e-6f);
        rb = 1.f / (fmaxf(fabsf(den_b + nq_s[tb]), em_s[tb]) + 1e-6f);
    }
    float* dst = o_raw + (size_t)row0 * nH * dv + (size_t)head * dv + sl * DVS;
#pragma unroll
    for (int j = 0; j < DVS / 8; ++j) {
        if (ta < n) *reinterpret_cast<float2*>(dst + (size_t)ta * nH * dv + j * 8 + 2 * tq) = make_float2(o[j][0] * ra, o[j][1] * ra);
        if (tb < n) *reinterpret_cast<float2*>(dst + (size_t)tb * nH * dv + j * 8 + 2 * tq) = make_float2(o[j][2] * rb, o[j][3] * rb);
    }
}

// -------------------------------------------------------------------------------------------- launchers
NG_EXPORT int ng_dl_slices(int dv) { return (dv + DL_SLICE - 1) / DL_SLICE; }

// Whether the chunk-by-chunk kernels take these head sizes.
NG_EXPORT int ng_dl_chunked_takes(int dk, int dv) { return dk > 0 && dv > 0 && dk % 16 == 0 && dv % 16 == 0 && dk <= 256; }

template <typename T, int MODE>
static int dl_step(const void* x, const float* gates, const float* gate_bias, const float* decay, float cap, float* state,
                   float* nm, float* o_raw, const int* cu_q, const int* ctx, const int* slots, int n_entries, DlGeom geo,
                   cudaStream_t stream) {
    const int G = (geo.dk + DL_ROWS - 1) / DL_ROWS;
    const size_t smem = ((size_t)DL_TOKENS * (2 * geo.dk + 32 + G * 32 + G)) * sizeof(float);
    static bool attr = false;
    if (!attr) {
        if (cudaFuncSetAttribute(dl_step_kernel<T, MODE>, cudaFuncAttributeMaxDynamicSharedMemorySize, 96 * 1024) != cudaSuccess)
            return NG_LAUNCH_FAILED;
        attr = true;
    }
    const dim3 grid(n_entries, geo.nH, ng_dl_slices(geo.dv));
    NG_LAUNCH((dl_step_kernel<T, MODE>), grid, 32 * G, smem, stream, (const T*)x, gates, gate_bias, decay, cap, state, nm, o_raw,
              cu_q, ctx, slots, geo);
    return ng_launch_status();
}

// Token by token.  x [n_rows, 2 nH (dk + dv)]; lightning (gates null): decay [nH][DC + 1], the powers of every head's
// decay; mLSTM: gates [n_rows, 2 nH] float32
// preactivations i | f, or g_parts partial sums of them g_stride elements apart, gate_bias [2 nH], nm_state [slots, nH, ng_dl_slices(dv), dk + 1].  o_raw float32 [n_rows, nH dv].
NG_EXPORT int ng_dl_step(const void* x, const float* gates, const float* gate_bias, const float* decay, float cap,
                         float* state, float* nm_state, float* o_raw, const int* cu_q, const int* ctx_before,
                         const int* slots, int n_entries, int nH, int dk, int dv, int g_parts, long long g_stride,
                         int act_bf16, cudaStream_t stream) {
    if (n_entries <= 0) return NG_OK;
    if (g_parts < 1) return NG_BAD_SIZE;
    if (nH <= 0 || nH > 65535 || dk <= 0 || dk > DL_ROWS * DL_MAX_WARPS || dv <= 0 || ng_dl_slices(dv) > 65535 || !state || !o_raw)
        return NG_BAD_SIZE;
    if (gates ? (!gate_bias || !nm_state || !(cap > 0.f)) : !decay) return NG_BAD_SIZE;
    const DlGeom geo{nH, dk, dv, g_parts, (size_t)g_stride};
#define DL_STEP(TT, MM) dl_step<TT, MM>(x, gates, gate_bias, decay, cap, state, nm_state, o_raw, cu_q, ctx_before, slots, n_entries, geo, stream)
    if (act_bf16) return gates ? DL_STEP(bf16, DL_MLSTM) : DL_STEP(bf16, DL_LIGHTNING);
    return gates ? DL_STEP(float, DL_MLSTM) : DL_STEP(float, DL_LIGHTNING);
}

// float32 values of scratch of ng_dl_chunked
NG_EXPORT long long ng_dl_chunked_scratch(int n_rows, int n_entries, int nH, int dk, int dv) {
    const long long slots = (long long)n_rows / DC + n_entries + 1;
    return slots * nH * ((long long)dk * dv + dk + 2) + (long long)n_rows * nH * 4 + 8;
}

template <int MODE, int DVS>
static int dl_chunked(const bf16* x, const float* gates, const float* gate_bias, const float* decay, float cap, float* state,
                      float* nm, float* o_raw, float* scratch, const int* cu_q, const int* ctx, const int* slots, int n_entries,
                      int n_rows, int max_q, DlGeom geo, cudaStream_t stream) {
    const size_t n_slots = (size_t)n_rows / DC + n_entries + 1;
    // 16-byte pieces first: per-token gates, then U, n and the chunks' numbers
    float4* tok = reinterpret_cast<float4*>(scratch);
    float* u = scratch + (size_t)n_rows * geo.nH * 4;
    float* un = u + n_slots * geo.nH * geo.dk * geo.dv;
    float2* chk = reinterpret_cast<float2*>(un + n_slots * geo.nH * geo.dk);
    const size_t sl = dl_local_smem<DVS>(geo.dk), so = dl_out_smem<DVS>(geo.dk);
    static bool attr = false;
    if (!attr) {
        if (cudaFuncSetAttribute(dl_local_kernel<MODE, DVS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess ||
            cudaFuncSetAttribute(dl_out_kernel<MODE, DVS>, cudaFuncAttributeMaxDynamicSharedMemorySize, 200 * 1024) != cudaSuccess)
            return NG_LAUNCH_FAILED;
        attr = true;
    }
    const int step_slices = ng_dl_slices(geo.dv);
    const dim3 grid((max_q + DC - 1) / DC, n_entries, geo.nH * (geo.dv / DVS));
    const int elems = geo.dk * geo.dv + (MODE == DL_MLSTM ? geo.dk : 0);
    const dim3 sgrid((elems / 4 + 255) / 256, n_entries, geo.nH);
    if (grid.y > 65535 || grid.z > 65535 || so > 200 * 1024) return NG_BAD_SIZE;
    if (MODE == DL_MLSTM)
        NG_LAUNCH((dl_gates_kernel), dim3(n_entries, geo.nH), 1024, 0, stream, gates, gate_bias, cap, tok, chk, nm, cu_q, ctx, slots,
                  geo, step_slices);
    NG_LAUNCH((dl_local_kernel<MODE, DVS>), grid, DC_THREADS, sl, stream, x, (const float4*)tok, decay, u, un, cu_q, geo);
    NG_LAUNCH((dl_scan_kernel<MODE>), sgrid, 256, 0, stream, u, un, state, nm, decay, (const float2*)chk, cu_q, ctx, slots, geo, step_slices);
    NG_LAUNCH((dl_out_kernel<MODE, DVS>), grid, DC_THREADS, so, stream, x, (const float4*)tok, (const float2*)chk, decay,
              (const float*)u, (const float*)un, o_raw, cu_q, geo);
    return ng_launch_status();
}

// As ng_dl_step for bfloat16 steps with long portions (max_q bounds the longest); scratch: ng_dl_chunked_scratch float32
// values, 16-byte aligned.
NG_EXPORT int ng_dl_chunked(const void* x, const float* gates, const float* gate_bias, const float* decay, float cap,
                            float* state, float* nm_state, float* o_raw, float* scratch, const int* cu_q,
                            const int* ctx_before, const int* slots, int n_entries, int n_rows, int max_q, int nH, int dk,
                            int dv, int g_parts, long long g_stride, cudaStream_t stream) {
    if (n_entries <= 0 || n_rows <= 0 || max_q <= 0) return NG_OK;
    if (g_parts < 1) return NG_BAD_SIZE;
    if (nH <= 0 || !ng_dl_chunked_takes(dk, dv) || !state || !o_raw || !scratch || ((uintptr_t)scratch & 15) ||
        ((uintptr_t)x & 15) || ((uintptr_t)state & 15) || ((uintptr_t)o_raw & 7))
        return NG_BAD_SIZE;
    if (gates ? (!gate_bias || !nm_state || !(cap > 0.f)) : !decay) return NG_BAD_SIZE;
    const DlGeom geo{nH, dk, dv, g_parts, (size_t)g_stride};
    const int dvs = dv % 64 == 0 ? 64 : dv % 32 == 0 ? 32 : 16;
#define DL_CHUNKED(MM, SS) dl_chunked<MM, SS>((const bf16*)x, gates, gate_bias, decay, cap, state, nm_state, o_raw, scratch, cu_q, \
                                              ctx_before, slots, n_entries, n_rows, max_q, geo, stream)
    if (gates) return dvs == 64 ? DL_CHUNKED(DL_MLSTM, 64) : dvs == 32 ? DL_CHUNKED(DL_MLSTM, 32) : DL_CHUNKED(DL_MLSTM, 16);
    return dvs == 64 ? DL_CHUNKED(DL_LIGHTNING, 64) : dvs == 32 ? DL_CHUNKED(DL_LIGHTNING, 32) : DL_CHUNKED(DL_LIGHTNING, 16);
}

// o_raw float32 [n_rows, width] -> out (rows ldo apart), groups of `group` columns normed; gate rows ldg apart.
NG_EXPORT int ng_dl_finish(const float* o_raw, const void* gate, const float* w, void* out, const int* row_entry, int n_rows,
                           int width, int group, int ldg, int ldo, float eps, float scale, int act_bf16, cudaStream_t stream) {
    if (n_rows <= 0) return NG_OK;
    if (width <= 0 || group <= 0 || width % group || ldg < width || ldo < width) return NG_BAD_SIZE;
    const size_t pair = act_bf16 ? 8 : 16;             // bytes of four activations
    const bool vec = group % 4 == 0 && ldg % 4 == 0 && ldo % 4 == 0 && ((uintptr_t)o_raw & 15) == 0 && ((uintptr_t)w & 15) == 0 &&
                     (uintptr_t)gate % pair == 0 && (uintptr_t)out % pair == 0;
#define DL_FINISH_VEC(TT, WH, NV, GRID, THREADS)                                                                          \
    NG_LAUNCH((dl_finish_vec_kernel<TT, WH, NV>), (GRID), (THREADS), 0, stream, o_raw, (const TT*)gate, w, (TT*)out, row_entry, n_rows, \
              width, group, ldg, ldo, eps, scale)
    if (vec && group == width && width <= 8192) {      // a block per row
        const int threads = width >= 2048 ? 512 : (width / 4 + 31) / 32 * 32;
        const int nv = (width + 4 * threads - 1) / (4 * threads);
        if (act_bf16) { if (nv <= 1) DL_FINISH_VEC(bf16, true, 1, n_rows, threads); else if (nv <= 2) DL_FINISH_VEC(bf16, true, 2, n_rows, threads); else DL_FINISH_VEC(bf16, true, 4, n_rows, threads); }
        else { if (nv <= 1) DL_FINISH_VEC(float, true, 1, n_rows, threads); else if (nv <= 2) DL_FINISH_VEC(float, true, 2, n_rows, threads); else DL_FINISH_VEC(float, true, 4, n_rows, threads); }
        return ng_launch_status();
    }
    if (vec && group < width && group <= 512) {        // a warp per (row, head)
        const size_t units = (size_t)n_rows * (width / group);
        const unsigned blocks = (unsigned)((units + 3) / 4);
        const int nv = (group + 127) / 128;
        if (act_bf16) { if (nv <= 1) DL_FINISH_VEC(bf16, false, 1, blocks, 128); else if (nv <= 2) DL_FINISH_VEC(bf16, false, 2, blocks, 128); else DL_FINISH_VEC(bf16, false, 4, blocks, 128); }
        else { if (nv <= 1) DL_FINISH_VEC(float, false, 1, blocks, 128); else if (nv <= 2) DL_FINISH_VEC(float, false, 2, blocks, 128); else DL_FINISH_VEC(float, false, 4, blocks, 128); }
        return ng_launch_status();
    }
    if (act_bf16)
        NG_LAUNCH((dl_finish_kernel<bf16>), n_rows, 256, 0, stream, o_raw, (const bf16*)gate, w, (bf16*)out, row_entry, width, group, ldg, ldo, eps, scale);
    else
        NG_LAUNCH((dl_finish_kernel<float>), n_rows, 256, 0, stream, o_raw, (const float*)gate, w, (float*)out, row_entry, width, group, ldg, ldo, eps, scale);
    return ng_launch_status();
}
