// Recurrences that run element by element:  S_t = a_t S_(t-1) + b_t  per channel, S from the request's state row (float32,
// zero in a fresh slot), out_t = S_t * gate_t.  Two kinds of a, b and gate (LS_*), each made from a product's columns:
//
//   LS_MIN_GRU   z = sigmoid(zr + z_b), u = xr + x_b;  a = 1 - z, b = z c(u), c(u) = u + 1/2 for u >= 0, sigmoid(u) else;
//                gate = silu(gr).  zr, xr, gr: columns 0, C, 2C of `proj`.
//   LS_GATED_LRU r = sigmoid(zr + r_b), i = sigmoid(zi + i_b) with zr, zi from `gates` [T, blocks of (K of r | K of i)]
//                (float32); log a = decay r (decay <= 0 per channel), a = exp(log a), b = sqrt(1 - a^2) i u with u from
//                `conv` [T, C]; gate = gelu_tanh(yr + y_b), yr from column 0 of `proj`.
//
// Float32 between load and store; bfloat16 steps take the special-function unit's exponential and division (a few units in the
// last place of float32), float32 steps the library's.  A request's tokens lie at rows cu[b] .. cu[b+1]-1.
// Steps of single tokens: a thread per (request, channel).  Else a block owns 32 channels and walks its tokens LS_TOKENS at a
// time: each of LS_SEG threads of a channel folds LS_RUN neighbouring tokens into one pair (A, B) with S_end = A S_begin + B,
// composes the pairs before its own and all of them through shared memory, and walks its tokens again, in registers, from
// its own S_begin.  Long portions: up to LS_CLUSTER blocks of a cluster take neighbouring stretches of LS_TOKENS tokens, read one
// another's composed pairs through the cluster's shared memory and chain them in their order from the carried state, so one
// read of the inputs serves all SMs.  A stretch's pair is composed the same way whoever makes it: the results do not depend
// on the number of blocks, only on where a portion starts.
#include "common.cuh"

#define LS_MIN_GRU 0
#define LS_GATED_LRU 1
#define LS_RUN 8
#define LS_SEG 16
#define LS_CH 32
#define LS_TOKENS (LS_SEG * LS_RUN)
#define LS_CLUSTER 8

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

template <bool FAST> __device__ __forceinline__ float ls_exp(float x) { return FAST ? __expf(x) : expf(x); }
template <bool FAST> __device__ __forceinline__ float ls_inv(float x) { return FAST ? __fdividef(1.f, x) : 1.f / x; }
template <bool FAST> __device__ __forceinline__ float ls_sigmoid(float x) { return ls_inv<FAST>(1.f + ls_exp<FAST>(-x)); }
// sqrt(1 - a^2) for a = exp(la), la <= 0; near la = 0 from the series of 1 - e^(2 la), which does not cancel
template <bool FAST> __device__ __forceinline__ float ls_input_scale(float la, float a) {
    if (!FAST) return sqrtf(-expm1f(2.f * la));
    const float y = -2.f * la;
    const float series = y * (1.f - y * (1.f / 2.f) * (1.f - y * (1.f / 3.f) * (1.f - y * (1.f / 4.f) * (1.f - y * (1.f / 5.f) * (1.f - y * (1.f / 6.f))))));
    const float q = y < 0.25f ? series : 1.f - a * a;
    return q > 0.f ? q * rsqrtf(q) : 0.f;
}

template <typename T, int KIND>
struct LsRaw {
    float v[KIND == LS_MIN_GRU ? 3 : 4];
    __device__ __forceinline__ void load(const LinearScan<T>& p, size_t row, int c, int gc) {
        const T* pr = p.proj + row * p.ld + c;
        if (KIND == LS_MIN_GRU) {
            v[0] = to_f32(pr[0]); v[1] = to_f32(pr[p.C]); v[2] = to_f32(pr[2 * (size_t)p.C]);
        } else {
            const float* g = p.gates + row * p.gates_ld + gc;
            v[0] = g[0]; v[1] = g[p.K]; v[2] = to_f32(p.conv[row * p.conv_ld + c]); v[KIND == LS_MIN_GRU ? 0 : 3] = to_f32(pr[0]);
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
    template <typename T> __device__ __forceinline__ void make(const LsRaw<T, KIND>& r, float& a, float& b, float& g) const {
        if (KIND == LS_MIN_GRU) {
            const float z = r.v[0] + b0, u = r.v[1] + b1;
            const float e = ls_exp<FAST>(-fabsf(z)), big = ls_inv<FAST>(1.f + e), small = e * big;      // sigmoid of |z| and of -|z|
            a = z >= 0.f ? small : big;
            b = (z >= 0.f ? big : small) * (u >= 0.f ? u + 0.5f : ls_sigmoid<FAST>(u));
            g = r.v[2] * ls_sigmoid<FAST>(r.v[2]);
        } else {
            const float la = decay * ls_sigmoid<FAST>(r.v[0] + b0);
            a = ls_exp<FAST>(la);
            b = ls_input_scale<FAST>(la, a) * ls_sigmoid<FAST>(r.v[1] + b1) * r.v[2];
            const float y = r.v[KIND == LS_MIN_GRU ? 0 : 3] + b2;
            g = y * ls_sigmoid<FAST>(2.f * 0.7978845608028654f * (y + 0.044715f * y * y * y));    // (1 + tanh(w)) / 2 = sigmoid(2 w)
        }
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
    LsRaw<T, KIND> r;
    r.load(p, row, c, ls_gate_column(p, c));
    float S = *st, a, bb, g;
    ch.make(r, a, bb, g);
    S = a * S + bb;
    *st = S;
    p.out[(size_t)row * p.C + c] = from_f32<T>(S * g);
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
template <typename T, int KIND, bool CL>
__global__ void __launch_bounds__(LS_CH * LS_SEG)
linear_scan_kernel(LinearScan<T> p) {
    __shared__ float2 s_pair[LS_SEG][LS_CH];
    __shared__ float2 s_total[2][LS_CH];                              // (CL) this block's composed pair, two stretches in turn
    pdl_launch_dependents();
    const int b = blockIdx.y, lane = threadIdx.x % LS_CH, seg = threadIdx.x / LS_CH;
    const int rank = CL ? blockIdx.z : 0, blocks = CL ? gridDim.z : 1;
    const int c = blockIdx.x * LS_CH + lane;
    const int s0 = p.cu[b], n = p.cu[b + 1] - s0;
    const bool live = c < p.C;
    const int cc = live ? c : p.C - 1, gc = ls_gate_column(p, cc);
    LsChannel<KIND, sizeof(T) == 2> ch;
    ch.load(p, cc);
    pdl_wait();
    if (n <= 0) return;                                               // (all blocks of a cluster serve one request)
    float* st = p.state + (long long)p.slots[b] * p.state_stride + cc;
    float carry = *st;
    int turn = 0;
    for (int base = 0; base < n; base += blocks * LS_TOKENS, turn ^= 1) {
        const int t0 = base + rank * LS_TOKENS + seg * LS_RUN;
        LsRaw<T, KIND> raw[LS_RUN];
#pragma unroll
        for (int j = 0; j < LS_RUN; ++j)
            if (t0 + j < n) raw[j].load(p, (size_t)(s0 + t0 + j), cc, gc);
        float a[LS_RUN], x[LS_RUN], g[LS_RUN], A = 1.f, B = 0.f;
#pragma unroll
        for (int j = 0; j < LS_RUN; ++j) {
            a[j] = 1.f; x[j] = 0.f; g[j] = 0.f;
            if (t0 + j < n) ch.make(raw[j], a[j], x[j], g[j]);
            A *= a[j];
            B = a[j] * B + x[j];
        }
        s_pair[seg][lane] = make_float2(A, B);
        __syncthreads();
        float PA = 1.f, PB = 0.f, TA = 1.f, TB = 0.f;                 // the pairs before this segment, and all of them
#pragma unroll
        for (int s = 0; s < LS_SEG; ++s) {
            if (s == seg) { PA = TA; PB = TB; }
            const float2 v = s_pair[s][lane];
            TA *= v.x;
            TB = v.x * TB + v.y;
        }
        float begin = carry;
        if (CL) {
            if (seg == 0) s_total[turn][lane] = make_float2(TA, TB);
            ls_cluster_sync();
            float S = carry;
            for (int r = 0; r < blocks; ++r) {
                if (r == rank) begin = S;
                const float2 v = ls_ld_cluster(ls_map_to_rank(&s_total[turn][lane], (unsigned)r));
                S = v.x * S + v.y;
            }
            carry = S;
        } else {
            carry = TA * carry + TB;
        }
        float S = PA * begin + PB;
#pragma unroll
        for (int j = 0; j < LS_RUN; ++j) {
            S = a[j] * S + x[j];
            if (live && t0 + j < n) p.out[(size_t)(s0 + t0 + j) * p.C + c] = from_f32<T>(S * g[j]);
        }
        __syncthreads();                                              // the pairs may be written again
    }
    // every thread that reads a state read it before its first barrier
    if (live && seg == 0 && rank == 0) *st = carry;
    if (CL) ls_cluster_sync();                                        // no block leaves while another may still read its pairs
}

template <typename T, int KIND>
static int launch_linear_scan(const LinearScan<T>& p, int B, int longest, cudaStream_t s) {
    if (longest == 1) return vl_launch(linear_step_kernel<T, KIND>, dim3((p.C + 127) / 128, B), dim3(128), 0, s, p);
    const dim3 threads(LS_CH * LS_SEG);
    int blocks = (longest + LS_TOKENS - 1) / LS_TOKENS;
    if (blocks > LS_CLUSTER) blocks = LS_CLUSTER;
    if (blocks <= 1) return vl_launch(linear_scan_kernel<T, KIND, false>, dim3((p.C + LS_CH - 1) / LS_CH, B), threads, 0, s, p);
    cudaLaunchConfig_t cfg = {};
    cfg.gridDim = dim3((p.C + LS_CH - 1) / LS_CH, B, blocks);
    cfg.blockDim = threads;
    cfg.stream = s;
    cudaLaunchAttribute attr[1];
    attr[0].id = cudaLaunchAttributeClusterDimension;
    attr[0].val.clusterDim.x = 1; attr[0].val.clusterDim.y = 1; attr[0].val.clusterDim.z = blocks;
    cfg.attrs = attr;
    cfg.numAttrs = 1;                                                 // (a step that long is launched the plain way, without dependents)
    return (int)cudaLaunchKernelEx(&cfg, linear_scan_kernel<T, KIND, true>, p);
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
