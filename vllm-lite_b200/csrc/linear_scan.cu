// Recurrences that run element by element:  S_t = a_t S_(t-1) + b_t  per channel, S from the request's state row (float32,
// zero in a fresh slot), out_t = S_t * gate_t.  Two kinds of a, b and gate (LS_*), each made from a product's columns:
//
//   LS_MIN_GRU   z = sigmoid(zr + z_b), u = xr + x_b;  a = 1 - z, b = z c(u), c(u) = u + 1/2 for u >= 0, sigmoid(u) else;
//                gate = silu(gr).  zr, xr, gr: columns 0, C, 2C of `proj`.
//   LS_GATED_LRU r = sigmoid(zr + r_b), i = sigmoid(zi + i_b) with zr, zi from `gates` [T, blocks of (K of r | K of i)]
//                (float32); log a = decay r (decay <= 0 per channel), a = exp(log a), b = sqrt(1 - a^2) i u with u from
//                `conv` [T, C]; gate = gelu_tanh(yr + y_b), yr from column 0 of `proj`.
//
// Float32 between load and store; bfloat16 steps take the special-function unit's exponential, reciprocal and root (a few units
// in the last place of float32), float32 steps the library's.  A request's tokens lie at rows cu[b] .. cu[b+1]-1.
// Steps of single tokens: a thread per (request, channel).  Else a block owns 32 lanes of VEC channels (two where everything
// lies on even columns) and walks its tokens LS_TOKENS at a time: each of LS_SEG warps folds LS_RUN neighbouring tokens of every
// channel into one pair (A, B) with S_end = A S_begin + B; a thread per channel composes the pairs before every warp's and all
// of them; the warps walk their tokens again, in registers, from their own S_begin.  Long portions: up to LS_CLUSTER blocks of a
// cluster take neighbouring stretches of LS_TOKENS tokens, read one another's composed pairs through the cluster's shared
// memory and chain them in their order from the carried state, so one read of the inputs serves all SMs.  A stretch's pair is
// composed the same way whoever makes it: the results do not depend on the number of blocks, only on where a portion starts.
#include "common.cuh"

#define LS_MIN_GRU 0
#define LS_GATED_LRU 1
#define LS_RUN 4
#define LS_SEG 16
#define LS_LANES 32
#define LS_TOKENS (LS_SEG * LS_RUN)
#define LS_CLUSTER 8
#define LS_LOG2E 1.4426950408889634f

template <typename T>
struct LinearScan {
    const T* proj; int ld;                               // [T, ld]
    const T* conv; int conv_ld;                          // (LRU) [T, C]
    const float* gates; int gates_ld, K;                 // (LRU) [T, 2 C] in blocks of K
    const float* p0; const float* p1; const float* p2; const float* decay;   // biases per channel: z, x | r, i, y; (LRU) decay
    float* state; long long state_stride;
    const int* cu; const int* slots;
    T* out; int C;
};

__device__ __forceinline__ float ls_ex2(float x) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
__device__ __forceinline__ float ls_rcp(float x) {
    float y;
    asm("rcp.approx.ftz.f32 %0, %1;" : "=f"(y) : "f"(x));
    return y;
}
template <bool FAST> __device__ __forceinline__ float ls_exp(float x) { return FAST ? ls_ex2(x * LS_LOG2E) : expf(x); }
template <bool FAST> __device__ __forceinline__ float ls_inv(float x) { return FAST ? ls_rcp(x) : 1.f / x; }
template <bool FAST> __device__ __forceinline__ float ls_sigmoid(float x) { return ls_inv<FAST>(1.f + ls_exp<FAST>(-x)); }
// sqrt(1 - a^2) for a = exp(la), la <= 0; near la = 0 from the series of 1 - e^(2 la), which does not cancel
template <bool FAST> __device__ __forceinline__ float ls_input_scale(float la, float a) {
    if (!FAST) return sqrtf(-expm1f(2.f * la));
    const float y = -2.f * la;
    const float series = y * (1.f - y * (1.f / 2.f) * (1.f - y * (1.f / 3.f) * (1.f - y * (1.f / 4.f) * (1.f - y * (1.f / 5.f)))));
    const float q = y < 0.125f ? series : 1.f - a * a;
    float s;
    asm("sqrt.approx.ftz.f32 %0, %1;" : "=f"(s) : "f"(q));
    return s;
}

// VEC neighbouring columns as float32
template <int VEC> __device__ __forceinline__ void ls_load(const float* p, float (&v)[VEC]) {
    if (VEC == 2) {
        const float2 q = *reinterpret_cast<const float2*>(p);
        v[0] = q.x; v[VEC - 1] = q.y;
    } else {
        v[0] = p[0];
    }
}
template <int VEC> __device__ __forceinline__ void ls_load(const bf16* p, float (&v)[VEC]) {
    if (VEC == 2) {
        const unsigned q = *reinterpret_cast<const unsigned*>(p);
        v[0] = __uint_as_float(q << 16); v[VEC - 1] = __uint_as_float(q & 0xffff0000u);
    } else {
        v[0] = __bfloat162float(p[0]);
    }
}
template <int VEC> __device__ __forceinline__ void ls_store(float* p, const float (&v)[VEC]) {
    if (VEC == 2) *reinterpret_cast<float2*>(p) = make_float2(v[0], v[VEC - 1]); else p[0] = v[0];
}
template <int VEC> __device__ __forceinline__ void ls_store(bf16* p, const float (&v)[VEC]) {
    if (VEC == 2) *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(v[0], v[VEC - 1]); else p[0] = __float2bfloat16_rn(v[0]);
}

// The values of a token's channels: what a and b are made of, and the output gate's.
template <typename T, int KIND, int VEC>
struct LsRaw {
    float p[VEC], q[VEC], u[VEC], g[VEC];                            // z, x, - | r, i, conv; the gate
    // pr, gt, cv: the token's rows at the thread's first channel
    __device__ __forceinline__ void load(const T* pr, const float* gt, const T* cv, int C, int K) {
        if (KIND == LS_MIN_GRU) {
            ls_load<VEC>(pr, p); ls_load<VEC>(pr + C, q); ls_load<VEC>(pr + 2 * C, g);
        } else {
            ls_load<VEC>(gt, p); ls_load<VEC>(gt + K, q); ls_load<VEC>(cv, u); ls_load<VEC>(pr, g);
        }
    }
};
// the channel's constants
template <int KIND, bool FAST>
struct LsChannel {
    float b0, b1, b2, decay;
    template <typename T> __device__ __forceinline__ void load(const LinearScan<T>& p, int c) {
        b0 = p.p0 ? p.p0[c] : 0.f; b1 = p.p1 ? p.p1[c] : 0.f;
        b2 = (KIND == LS_GATED_LRU && p.p2) ? p.p2[c] : 0.f;
        decay = KIND == LS_GATED_LRU ? p.decay[c] : 0.f;
    }
    __device__ __forceinline__ void make(float p, float q, float u, float& a, float& b) const {
        if (KIND == LS_MIN_GRU) {
            const float z = p + b0, x = q + b1;
            const float e = ls_exp<FAST>(-fabsf(z)), big = ls_inv<FAST>(1.f + e), small = e * big;      // sigmoid of |z| and of -|z|
            a = z >= 0.f ? small : big;
            b = (z >= 0.f ? big : small) * (x >= 0.f ? x + 0.5f : ls_sigmoid<FAST>(x));
        } else {
            const float la = decay * ls_sigmoid<FAST>(p + b0);
            a = ls_exp<FAST>(la);
            b = ls_input_scale<FAST>(la, a) * ls_sigmoid<FAST>(q + b1) * u;
        }
    }
    __device__ __forceinline__ float gate(float g) const {
        if (KIND == LS_MIN_GRU) return g * ls_sigmoid<FAST>(g);
        const float y = g + b2;
        return y * ls_sigmoid<FAST>(y * (2.f * 0.7978845608028654f + 2.f * 0.7978845608028654f * 0.044715f * y * y));     // (1 + tanh(w)) / 2 = sigmoid(2 w)
    }
};
template <typename T>
__device__ __forceinline__ int ls_gate_column(const LinearScan<T>& p, int c) {
    return p.K > 0 ? c / p.K * 2 * p.K + c % p.K : 0;
}

template <typename T, int KIND>
__global__ void __launch_bounds__(128)
linear_step_kernel(LinearScan<T> p) {
    pdl_launch_dependents();
    const int b = blockIdx.y, c = blockIdx.x * 128 + threadIdx.x;
    const int row = p.cu[b], n = p.cu[b + 1] - row;
    LsChannel<KIND, sizeof(T) == 2> ch;
    if (c < p.C) ch.load(p, c);
    pdl_wait();
    if (n <= 0 || c >= p.C) return;
    float* st = p.state + (long long)p.slots[b] * p.state_stride + c;
    LsRaw<T, KIND, 1> r;
    r.load(p.proj + (size_t)row * p.ld + c, p.gates + (size_t)row * p.gates_ld + ls_gate_column(p, c), p.conv + (size_t)row * p.conv_ld + c, p.C, p.K);
    float S = *st, a, bb;
    ch.make(r.p[0], r.q[0], r.u[0], a, bb);
    S = a * S + bb;
    *st = S;
    p.out[(size_t)row * p.C + c] = from_f32<T>(S * ch.gate(r.g[0]));
}

__device__ __forceinline__ unsigned ls_map_to_rank(const void* p, unsigned rank) {
    unsigned a;
    asm volatile("mapa.shared::cluster.u32 %0, %1, %2;" : "=r"(a) : "r"((unsigned)__cvta_generic_to_shared(p)), "r"(rank));
    return a;
}
__device__ __forceinline__ float2 ls_ld_cluster(unsigned addr) {
    float2 v;
    asm volatile("ld.shared::cluster.v2.f32 {%0, %1}, [%2];" : "=f"(v.x), "=f"(v.y) : "r"(addr) : "memory");
    return v;
}
__device__ __forceinline__ void ls_cluster_sync() {
    asm volatile("barrier.cluster.arrive.release.aligned;\n barrier.cluster.wait.acquire.aligned;" ::: "memory");
}

// CL: the blocks of a z row are one cluster
template <typename T, int KIND, int VEC, bool CL>
__global__ void __launch_bounds__(LS_LANES * LS_SEG, 2)
linear_scan_kernel(LinearScan<T> p) {
    __shared__ float2 s_pair[LS_SEG][VEC][LS_LANES];                  // every warp's pair, then the composed pairs before it
    __shared__ float2 s_total[2][VEC][LS_LANES];                      // the stretch's composed pair, two stretches in turn
    __shared__ float s_begin[VEC][LS_LANES];                          // the state the block's stretch begins with
    pdl_launch_dependents();
    const int b = blockIdx.y, lane = threadIdx.x % LS_LANES, seg = threadIdx.x / LS_LANES;
    const int rank = CL ? blockIdx.z : 0, blocks = CL ? gridDim.z : 1;
    const int c = (blockIdx.x * LS_LANES + lane) * VEC;
    const int s0 = p.cu[b], n = p.cu[b + 1] - s0;
    const bool live = c < p.C;
    const int cc = live ? c : p.C - VEC;
    LsChannel<KIND, sizeof(T) == 2> ch[VEC];
#pragma unroll
    for (int v = 0; v < VEC; ++v) ch[v].load(p, cc + v);
    pdl_wait();
    if (n <= 0) return;                                               // (all blocks of a cluster serve one request)
    const T* proj = p.proj + (size_t)s0 * p.ld + cc;
    const T* conv = KIND == LS_GATED_LRU ? p.conv + (size_t)s0 * p.conv_ld + cc : nullptr;
    const float* gates = KIND == LS_GATED_LRU ? p.gates + (size_t)s0 * p.gates_ld + ls_gate_column(p, cc) : nullptr;
    // threads 0 .. VEC * 32 - 1 chain the pairs of channel (v, lane) = (seg, lane) and carry its state
    float* st = p.state + (long long)p.slots[b] * p.state_stride + cc + min(seg, VEC - 1);
    float carry = seg < VEC ? *st : 0.f;
    int turn = 0;
    for (int base = 0; base < n; base += blocks * LS_TOKENS, turn ^= 1) {
        const int t0 = base + rank * LS_TOKENS + seg * LS_RUN, m = n - t0;       // (a warp's tokens; m may be 0 or less)
        LsRaw<T, KIND, VEC> raw[LS_RUN];
        {
            const size_t at = (size_t)min(t0, n - 1);                 // past the end: some row of the request, never used
            const T* pr = proj + at * p.ld;
            const T* cv = conv + at * p.conv_ld;
            const float* gt = gates + at * p.gates_ld;
#pragma unroll
            for (int j = 0; j < LS_RUN; ++j) {
                raw[j].load(pr, gt, cv, p.C, p.K);
                if (j + 1 < m) { pr += p.ld; cv += p.conv_ld; gt += p.gates_ld; }
            }
        }
        float a[LS_RUN][VEC], x[LS_RUN][VEC], A[VEC], B[VEC];
#pragma unroll
        for (int v = 0; v < VEC; ++v) { A[v] = 1.f; B[v] = 0.f; }
#pragma unroll
        for (int j = 0; j < LS_RUN; ++j)
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                ch[v].make(raw[j].p[v], raw[j].q[v], raw[j].u[v], a[j][v], x[j][v]);
                if (j >= m) { a[j][v] = 1.f; x[j][v] = 0.f; }
                A[v] *= a[j][v];
                B[v] = a[j][v] * B[v] + x[j][v];
            }
#pragma unroll
        for (int v = 0; v < VEC; ++v) s_pair[seg][v][lane] = make_float2(A[v], B[v]);
        __syncthreads();
        float2 total = make_float2(1.f, 0.f);
        if (seg < VEC) {                                              // a warp per v
            float2 w[LS_SEG];
#pragma unroll
            for (int s = 0; s < LS_SEG; ++s) w[s] = s_pair[s][seg][lane];
#pragma unroll
            for (int s = 0; s < LS_SEG; ++s) {
                s_pair[s][seg][lane] = total;
                total = make_float2(w[s].x * total.x, w[s].x * total.y + w[s].y);
            }
            if (CL) s_total[turn][seg][lane] = total;
        }
        if (CL) ls_cluster_sync();
        if (seg < VEC) {
            float S = carry, begin = carry;
            if (CL) {
                float2 w[LS_CLUSTER];
#pragma unroll
                for (int k = 0; k < LS_CLUSTER; ++k)                  // all loads first: they are in flight together
                    if (k < blocks) w[k] = ls_ld_cluster(ls_map_to_rank(&s_total[turn][seg][lane], (unsigned)k));
#pragma unroll
                for (int k = 0; k < LS_CLUSTER; ++k)
                    if (k < blocks) {
                        if (k == rank) begin = S;
                        S = w[k].x * S + w[k].y;
                    }
            } else {
                S = total.x * S + total.y;
            }
            carry = S;
            s_begin[seg][lane] = begin;
        }
        __syncthreads();
        float S[VEC];
#pragma unroll
        for (int v = 0; v < VEC; ++v) {
            const float2 w = s_pair[seg][v][lane];                    // (rewritten by this thread alone before the next barrier)
            S[v] = w.x * s_begin[v][lane] + w.y;
        }
        T* out = p.out + (size_t)(s0 + t0) * p.C + c;
#pragma unroll
        for (int j = 0; j < LS_RUN; ++j) {
            float o[VEC];
#pragma unroll
            for (int v = 0; v < VEC; ++v) {
                S[v] = a[j][v] * S[v] + x[j][v];
                o[v] = S[v] * ch[v].gate(raw[j].g[v]);
            }
            if (live && j < m) ls_store<VEC>(out + (size_t)j * p.C, o);
        }
    }
    // every thread that reads a state read it before its first barrier
    if (live && seg < VEC && rank == 0) *st = carry;
    if (CL) ls_cluster_sync();                                        // no block leaves while another may still read its pairs
}

template <typename T, int KIND, int VEC>
static int launch_linear_portions(const LinearScan<T>& p, int B, int longest, cudaStream_t s) {
    const dim3 threads(LS_LANES * LS_SEG);
    const unsigned tiles = (unsigned)((p.C + LS_LANES * VEC - 1) / (LS_LANES * VEC));
    int blocks = (longest + LS_TOKENS - 1) / LS_TOKENS;
    if (blocks > LS_CLUSTER) blocks = LS_CLUSTER;
    if (blocks <= 1) return vl_launch(linear_scan_kernel<T, KIND, VEC, false>, dim3(tiles, B), threads, 0, s, p);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3(tiles, B, blocks);
    cfg.blockDim = threads;
    cfg.stream = s;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = 1; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = blocks;
    cfg.attrs = attr;
    cfg.numAttrs = 1;                                                 // (a step that long is launched the plain way, without dependents)
    return (int)cudaLaunchKernelEx(&cfg, linear_scan_kernel<T, KIND, VEC, true>, p);
}

template <typename T, int KIND>
static int launch_linear_scan(const LinearScan<T>& p, int B, int longest, cudaStream_t s) {
    if (longest == 1) return vl_launch(linear_step_kernel<T, KIND>, dim3((p.C + 127) / 128, B), dim3(128), 0, s, p);
    const bool even = ((p.C | p.ld | p.conv_ld | p.gates_ld | p.K) & 1) == 0 &&
                      (((uintptr_t)p.proj | (uintptr_t)p.conv | (uintptr_t)p.gates | (uintptr_t)p.out) & 7) == 0;
    return even ? launch_linear_portions<T, KIND, 2>(p, B, longest, s) : launch_linear_portions<T, KIND, 1>(p, B, longest, s);
}

// longest: a bound on the tokens one request brings (1: a step of single tokens)
extern "C" int vl_linear_scan(int kind, const void* proj, int ld, int dtype, const void* conv, int conv_ld, const float* gates,
                              int gates_ld, int K, const float* p0, const float* p1, const float* p2, const float* decay, float* state,
                              long long state_stride, const int* cu, const int* slots, int B, int longest, void* out, int C, void* stream) {
    if (B <= 0 || C <= 0) return VL_OK;
    if (kind != LS_MIN_GRU && kind != LS_GATED_LRU) return VL_ERR_ARGUMENT;
    if (state_stride < C || longest <= 0 || B > 65535) return VL_ERR_ARGUMENT;
    if (kind == LS_MIN_GRU && ld < 3 * C) return VL_ERR_ARGUMENT;
    if (kind == LS_GATED_LRU && (!conv || !gates || !decay || K <= 0 || C % K || ld < C || conv_ld < C || gates_ld < 2 * C)) return VL_ERR_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
#define LS_LAUNCH(TT)                                                                                                          \
    do {                                                                                                                       \
        const LinearScan<TT> a = {(const TT*)proj, ld, (const TT*)conv, conv_ld, gates, gates_ld, K, p0, p1, p2, decay, state, \
                                  state_stride, cu, slots, (TT*)out, C};                                                       \
        return kind == LS_MIN_GRU ? launch_linear_scan<TT, LS_MIN_GRU>(a, B, longest, s)                                       \
                                  : launch_linear_scan<TT, LS_GATED_LRU>(a, B, longest, s);                                    \
    } while (0)
    if (dtype == VL_F32) LS_LAUNCH(float);
    if (dtype == VL_BF16) LS_LAUNCH(bf16);
#undef LS_LAUNCH
    return VL_ERR_UNSUPPORTED;
}
