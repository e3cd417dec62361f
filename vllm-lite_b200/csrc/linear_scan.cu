// Recurrences that run element by element:  S_t = a_t S_(t-1) + b_t  per channel, S from the request's state row (float32,
// zero in a fresh slot), out_t = S_t * gate_t.  Two kinds of a, b and gate (LS_*), each made from a product's columns:
//
//   LS_MIN_GRU   z = sigmoid(zr + z_b), u = xr + x_b;  a = 1 - z, b = z c(u), c(u) = u + 1/2 for u >= 0, sigmoid(u) else;
//                gate = silu(gr).  zr, xr, gr: columns 0, C, 2C of `proj`.
//   LS_GATED_LRU r = sigmoid(zr + r_b), i = sigmoid(zi + i_b) with zr, zi from `gates` [T, blocks of (K of r | K of i)]
//                (float32); log a = decay r (decay <= 0 per channel), a = exp(log a), b = sqrt(1 - a^2) i u with u from
//                `conv` [T, C]; gate = gelu_tanh(yr + y_b), yr from column 0 of `proj`.
//
// Float32 between load and store.  A request's tokens lie at rows cu[b] .. cu[b+1]-1.  Steps of single tokens: a thread per
// (request, channel).  Else a block owns CH channels of one request and walks its tokens SEG * LS_RUN at a time: each of SEG
// threads of a channel folds LS_RUN neighbouring tokens into one pair (A, B) with S_end = A S_begin + B, the SEG pairs are
// chained from the carried state through shared memory, and each thread walks its tokens again from its own S_begin.  The
// raw values of the next stretch are loaded before this one is walked.  The order of the sums depends on the model's
// sizes and on where a portion starts, not on the batch.
#include "common.cuh"

#define LS_MIN_GRU 0
#define LS_GATED_LRU 1
#define LS_RUN 8

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

__device__ __forceinline__ float ls_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }

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
template <int KIND>
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
            const float e = expf(-fabsf(z)), big = 1.f / (1.f + e), small = e * big;      // sigmoid of |z| and of -|z|
            a = z >= 0.f ? small : big;
            b = (z >= 0.f ? big : small) * (u >= 0.f ? u + 0.5f : ls_sigmoid(u));
            g = r.v[2] / (1.f + expf(-r.v[2]));
        } else {
            const float la = decay * ls_sigmoid(r.v[0] + b0);
            a = expf(la);
            b = sqrtf(-expm1f(2.f * la)) * ls_sigmoid(r.v[1] + b1) * r.v[2];
            const float y = r.v[KIND == LS_MIN_GRU ? 0 : 3] + b2;
            g = 0.5f * y * (1.f + tanhf(0.7978845608028654f * (y + 0.044715f * y * y * y)));
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
    LsChannel<KIND> ch;
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

template <typename T, int KIND, int CH, int SEG>
__global__ void __launch_bounds__(CH * SEG)
linear_scan_kernel(LinearScan<T> p) {
    __shared__ float s_a[SEG][CH], s_b[SEG][CH];
    pdl_launch_dependents();
    const int b = blockIdx.y, lane = threadIdx.x % CH, seg = threadIdx.x / CH;
    const int c = blockIdx.x * CH + lane;
    const int s0 = p.cu[b], n = p.cu[b + 1] - s0;
    const bool live = c < p.C;
    const int cc = live ? c : p.C - 1, gc = ls_gate_column(p, cc);
    LsChannel<KIND> ch;
    ch.load(p, cc);
    pdl_wait();
    if (n <= 0) return;
    float* st = p.state + (long long)p.slots[b] * p.state_stride + cc;
    float carry = *st;
    LsRaw<T, KIND> raw[LS_RUN];
    auto fetch = [&](int t0) {
#pragma unroll
        for (int j = 0; j < LS_RUN; ++j)
            if (t0 + j < n) raw[j].load(p, (size_t)(s0 + t0 + j), cc, gc);
    };
    fetch(seg * LS_RUN);
    for (int base = 0; base < n; base += SEG * LS_RUN) {
        const int t0 = base + seg * LS_RUN;
        float a[LS_RUN], x[LS_RUN], g[LS_RUN], A = 1.f, B = 0.f;
#pragma unroll
        for (int j = 0; j < LS_RUN; ++j) {
            a[j] = 1.f; x[j] = 0.f; g[j] = 0.f;
            if (t0 + j < n) ch.make(raw[j], a[j], x[j], g[j]);
            A *= a[j];
            B = a[j] * B + x[j];
        }
        if (base + SEG * LS_RUN < n) fetch(t0 + SEG * LS_RUN);
        s_a[seg][lane] = A;
        s_b[seg][lane] = B;
        __syncthreads();
        float S = carry, mine = carry;
#pragma unroll
        for (int s = 0; s < SEG; ++s) {
            if (s == seg) mine = S;
            S = s_a[s][lane] * S + s_b[s][lane];
        }
        carry = S;
#pragma unroll
        for (int j = 0; j < LS_RUN; ++j) {
            mine = a[j] * mine + x[j];
            if (live && t0 + j < n) p.out[(size_t)(s0 + t0 + j) * p.C + c] = from_f32<T>(mine * g[j]);
        }
        __syncthreads();                                              // the pairs may be written again
    }
    if (live && seg == 0) *st = carry;                                // (read by every thread of the channel before the first barrier)
}

template <typename T, int KIND>
static int launch_linear_scan(const LinearScan<T>& p, int B, int longest, cudaStream_t s) {
    if (longest == 1) return vl_launch(linear_step_kernel<T, KIND>, dim3((p.C + 127) / 128, B), dim3(128), 0, s, p);
    // narrow models: fewer channels a block, so that one request's channels give the SMs their blocks
    if (p.C <= 4096) return vl_launch(linear_scan_kernel<T, KIND, 16, 32>, dim3((p.C + 15) / 16, B), dim3(512), 0, s, p);
    return vl_launch(linear_scan_kernel<T, KIND, 32, 16>, dim3((p.C + 31) / 32, B), dim3(512), 0, s, p);
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
