// The gated delta rule with ONE decay per head, for states of up to 128 x 128 numbers a head:
//     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q         then   out = rms_head(o) * norm * silu(gate)
// over the tokens that a step brings for every request (rows cu[b] .. cu[b+1]-1), from the state in the request's slot.
// q, k, v are columns of `qkv` (float32, what the short convolution leaves: q heads | k heads | v heads), the raw decay and
// the raw beta columns of the stacked product's rows, the gate another block of columns there.  k and q are made unit
// vectors (q times q_scale), g = exp(-exp(A_log) softplus(a + dt_bias)), beta = sigmoid(b).  Everything is float32: no product
// here runs in fewer bits.  A head's state lies row by row, [D][P].
//
//   vl_delta_step    portions of fewer than DELTA_MIN_CHUNK tokens (decoding): a block per (head, request) holds the whole state in
//                    registers (16-byte accesses, 64 KB in flight a block at 128 x 128).  One pass over the state and one
//                    sum across the block a token: with w = S^T k and r = S^T q of the old state,
//                    u = beta (v - g w) and o = g r + (k.q) u.
//   vl_delta_chunks  longer portions, in chunks of 64 tokens from the portion's start.  With l_t = log g_t, L its running sum inside
//                    the chunk and S_0 the state at its start, the u of a chunk solve a triangular system,
//                        u_t + sum_{s<t} A_ts u_s = beta_t (v_t - e^(L_t) S_0^T k_t),   A_ts = beta_t e^(L_t - L_s) k_t.k_s
//                        o_t = e^(L_t) S_0^T q_t + sum_{s<=t} e^(L_t - L_s) (q_t.k_s) u_s
//                        S_end = e^(L_64) S_0 + sum_s e^(L_64 - L_s) k_s u_s^T
//                    (the WY form of the delta rule).  Three launches: (1) per chunk and head, all at once: both 64 x 64 matrices
//                    and the system solved for the right sides [beta v | beta e^L k], giving U0 and W; (2) per head, tile
//                    of value columns and request, chunk after chunk: U = U0 - W S, S <- e^(L_64) S + K'^T U; (3) per chunk and head,
//                    all at once: the outputs, normed and gated.
// L is summed in double precision and kept as two floats, so that differences of it are exact however far it has fallen.
// The order of every sum depends on the sizes and on the place in the portion alone, not on what else the launch holds.
#include "common.cuh"

#define DC 64                         // tokens of a chunk
#define DELTA_MIN_CHUNK 16            // portions of fewer tokens are walked token by token
#define DELTA_MAX 128                 // most rows and columns of a head's state

__device__ __forceinline__ float dl_softplus(float x) { return x > 20.f ? x : log1pf(expf(x)); }
__device__ __forceinline__ float dl_sigmoid(float x) { return 1.f / (1.f + expf(-x)); }
__device__ __forceinline__ float dl_silu(float x) { return x / (1.f + expf(-x)); }
__device__ __forceinline__ void dl_copy16(void* smem, const void* gmem, bool valid) {
    const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
    const int bytes = valid ? 16 : 0;                             // 0: the 16 bytes become zeros
    asm volatile("cp.async.cg.shared.global [%0], [%1], 16, %2;" ::"r"(dst), "l"(gmem), "r"(bytes) : "memory");
}
__device__ __forceinline__ void dl_commit() { asm volatile("cp.async.commit_group;" ::: "memory"); }
template <int N> __device__ __forceinline__ void dl_wait() { asm volatile("cp.async.wait_group %0;" ::"n"(N) : "memory"); }
__device__ __forceinline__ float4 ld4(const float* p) { return *reinterpret_cast<const float4*>(p); }
__device__ __forceinline__ void st4(float* p, float4 v) { *reinterpret_cast<float4*>(p) = v; }
__device__ __forceinline__ float dot4(float4 a, float4 b) { return a.x * b.x + a.y * b.y + a.z * b.z + a.w * b.w; }

static bool delta_sizes_ok(int H, int G, int D, int P, int C) {
    return H > 0 && G > 0 && H % G == 0 && D > 0 && P > 0 && D <= DELTA_MAX && P <= DELTA_MAX && D % 4 == 0 && P % 4 == 0 &&
           C == 2 * G * D + H * P;
}

// ------------------------------------------------------------------------------------------ few tokens
#define STEP_ROWS 8                   // rows of the state a thread holds (four columns each)
// How the threads lie over a state of D rows and U = P / 4 units of four columns: a warp covers LU neighbouring units of 32 / LU rows,
// UG warps side by side cover the units, WR of them one under the other the rows (STEP_ROWS rows a thread).
struct StepShape { int LU, UG, WR; };
static inline StepShape step_shape(int D, int U) {
    int LU = 1;
    while (LU < U && LU < 8) LU <<= 1;
    const int rows = 32 / LU * STEP_ROWS;
    return StepShape{LU, (U + LU - 1) / LU, (D + rows - 1) / rows};
}
template <typename TP>
__global__ void __launch_bounds__(512, 2)
delta_step_kernel(const float* __restrict__ qkv, int C, const TP* __restrict__ proj, int ld, int a_col, int b_col, int gate_col,
                  const float* __restrict__ dt_bias, const float* __restrict__ A_log, float q_scale, float unit_eps,
                  const float* __restrict__ norm, float eps, float* __restrict__ state, long long state_stride,
                  const int* __restrict__ cu, const int* __restrict__ slots, TP* __restrict__ out, int H, int G, int D, int P,
                  int longest, int LU, int UG, int WR) {
    __shared__ __align__(16) float sq[DELTA_MAX], sk[DELTA_MAX], su[DELTA_MAX], part[2][4][DELTA_MAX];
    __shared__ float s_g, s_beta, s_qk;
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, b = blockIdx.y;
    const int s0 = cu[b], n = cu[b + 1] - s0;
    if (n <= 0 || n > longest) return;
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int U = P >> 2, RG = WR * (32 / LU);
    const int unit = (warp % UG) * LU + lane % LU, wr = warp / UG, rg = wr * (32 / LU) + lane / LU;
    const bool live = unit < U;
    float* S = state + (long long)slots[b] * state_stride + (size_t)h * D * P + 4 * unit;
    float4 s[STEP_ROWS];
#pragma unroll
    for (int i = 0; i < STEP_ROWS; ++i) {
        const int r = rg + RG * i;
        s[i] = (live && r < D) ? ld4(S + r * P) : make_float4(0.f, 0.f, 0.f, 0.f);
    }
    const int g = h / (H / G);
    for (int t = 0; t < n; ++t) {
        const float* row = qkv + (size_t)(s0 + t) * C;
        const TP* prow = proj + (size_t)(s0 + t) * ld;
        float4 v = make_float4(0.f, 0.f, 0.f, 0.f), z = v;
        if (warp == 0) {                                          // unit vectors, their product; what the epilogue will need
            float4 q = v, k = v;
            if (4 * lane < D) { q = ld4(row + (size_t)g * D + 4 * lane); k = ld4(row + (size_t)(G + g) * D + 4 * lane); }
            if (lane < U) {
                v = ld4(row + (size_t)2 * G * D + (size_t)h * P + 4 * lane);
                z = Quad<TP>::load(prow + gate_col + (size_t)h * P + 4 * lane);
            }
            const float qn = q_scale / sqrtf(warp_sum(dot4(q, q)) + unit_eps), kn = 1.f / sqrtf(warp_sum(dot4(k, k)) + unit_eps);
            q.x *= qn; q.y *= qn; q.z *= qn; q.w *= qn;
            k.x *= kn; k.y *= kn; k.z *= kn; k.w *= kn;
            if (4 * lane < D) { st4(sq + 4 * lane, q); st4(sk + 4 * lane, k); }
            const float qk = warp_sum(dot4(q, k));
            if (lane == 0) s_qk = qk;
        }
        if (tid == blockDim.x - 1) {                              // the two numbers of the head (the last warp, or the only one)
            s_g = expf(-expf(A_log[h]) * dl_softplus(to_f32(prow[a_col + h]) + dt_bias[h]));
            s_beta = dl_sigmoid(to_f32(prow[b_col + h]));
        }
        __syncthreads();
        float4 w = make_float4(0.f, 0.f, 0.f, 0.f), r4 = w;
#pragma unroll
        for (int i = 0; i < STEP_ROWS; ++i) {
            const int r = rg + RG * i;
            if (r < D) {
                const float kr = sk[r], qr = sq[r];
                w.x += s[i].x * kr; w.y += s[i].y * kr; w.z += s[i].z * kr; w.w += s[i].w * kr;
                r4.x += s[i].x * qr; r4.y += s[i].y * qr; r4.z += s[i].z * qr; r4.w += s[i].w * qr;
            }
        }
        for (int o = LU; o < 32; o <<= 1) {                       // the warp's rows of a unit
            w.x += __shfl_xor_sync(0xffffffffu, w.x, o); w.y += __shfl_xor_sync(0xffffffffu, w.y, o);
            w.z += __shfl_xor_sync(0xffffffffu, w.z, o); w.w += __shfl_xor_sync(0xffffffffu, w.w, o);
            r4.x += __shfl_xor_sync(0xffffffffu, r4.x, o); r4.y += __shfl_xor_sync(0xffffffffu, r4.y, o);
            r4.z += __shfl_xor_sync(0xffffffffu, r4.z, o); r4.w += __shfl_xor_sync(0xffffffffu, r4.w, o);
        }
        if (live && lane < LU) {
            st4(&part[0][wr][4 * unit], w);
            st4(&part[1][wr][4 * unit], r4);
        }
        __syncthreads();
        const float gt = s_g;
        if (warp == 0) {
            float4 u = make_float4(0.f, 0.f, 0.f, 0.f), o = u;
            if (lane < U) {
                for (int i = 0; i < WR; ++i) {
                    const float4 a = ld4(&part[0][i][4 * lane]), c = ld4(&part[1][i][4 * lane]);
                    u.x += a.x; u.y += a.y; u.z += a.z; u.w += a.w;
                    o.x += c.x; o.y += c.y; o.z += c.z; o.w += c.w;
                }
                const float be = s_beta, qk = s_qk;
                u.x = be * (v.x - gt * u.x); u.y = be * (v.y - gt * u.y); u.z = be * (v.z - gt * u.z); u.w = be * (v.w - gt * u.w);
                o.x = gt * o.x + qk * u.x; o.y = gt * o.y + qk * u.y; o.z = gt * o.z + qk * u.z; o.w = gt * o.w + qk * u.w;
                st4(su + 4 * lane, u);
            }
            __syncwarp();
            const float inv = 1.f / sqrtf(warp_sum(dot4(o, o)) / (float)P + eps);
            if (lane < U) {
                const float4 nw = ld4(norm + 4 * lane);
                Quad<TP>::store(out + (size_t)(s0 + t) * H * P + (size_t)h * P + 4 * lane,
                                make_float4(o.x * inv * nw.x * dl_silu(z.x), o.y * inv * nw.y * dl_silu(z.y),
                                            o.z * inv * nw.z * dl_silu(z.z), o.w * inv * nw.w * dl_silu(z.w)));
            }
        }
        __syncthreads();
        const float4 u = live ? ld4(su + 4 * unit) : make_float4(0.f, 0.f, 0.f, 0.f);
#pragma unroll
        for (int i = 0; i < STEP_ROWS; ++i) {
            const int r = rg + RG * i;
            if (r < D) {
                const float kr = sk[r];
                s[i].x = gt * s[i].x + kr * u.x; s[i].y = gt * s[i].y + kr * u.y;
                s[i].z = gt * s[i].z + kr * u.z; s[i].w = gt * s[i].w + kr * u.w;
            }
        }
        if (t + 1 < n) __syncthreads();                           // the next token's unit vectors take sq and sk
    }
#pragma unroll
    for (int i = 0; i < STEP_ROWS; ++i) {
        const int r = rg + RG * i;
        if (live && r < D) st4(S + r * P, s[i]);
    }
}

extern "C" int vl_delta_step(const float* qkv, int C, const void* proj, int dtype, int ld, int a_col, int b_col, int gate_col,
                             const float* dt_bias, const float* A_log, float q_scale, float unit_eps, const float* norm, float eps,
                             float* state, long long state_stride, const int* cu, const int* slots, int B, void* out, int H, int G,
                             int D, int P, int longest, void* stream) {
    if (B <= 0) return VL_OK;
    if (!delta_sizes_ok(H, G, D, P, C)) return VL_ERR_UNSUPPORTED;
    if (ld % 4 || gate_col % 4 || state_stride % 4 || (((uintptr_t)qkv | (uintptr_t)proj | (uintptr_t)state | (uintptr_t)out | (uintptr_t)norm) & 15))
        return VL_ERR_ARGUMENT;
    const StepShape sh = step_shape(D, P / 4);                    // (at most 16 warps, four rows of them)
    cudaStream_t s = (cudaStream_t)stream;
#define DELTA_STEP(TP)                                                                                                              \
    return vl_launch(delta_step_kernel<TP>, dim3(H, B), dim3(32 * sh.UG * sh.WR), 0, s, qkv, C, (const TP*)proj, ld, a_col, b_col, gate_col, \
                     dt_bias, A_log, q_scale, unit_eps, norm, eps, state, state_stride, cu, slots, (TP*)out, H, G, D, P, longest,  \
                     sh.LU, sh.UG, sh.WR)
    if (dtype == VL_F32) DELTA_STEP(float);
    if (dtype == VL_BF16) DELTA_STEP(bf16);
#undef DELTA_STEP
    return VL_ERR_UNSUPPORTED;
}

// ------------------------------------------------------------------------------------------ chunks: which is whose
__device__ __forceinline__ int dl_chunks_of(const int* cu, int b, int B) {
    const int n = b < B ? cu[b + 1] - cu[b] : 0;
    return n >= DELTA_MIN_CHUNK ? (n + DC - 1) / DC : 0;
}
// Chunk number `idx` of the launch: request b and its chunk c.  Called by whole warps; false beyond the last chunk.
__device__ __forceinline__ bool dl_find(const int* cu, int B, int idx, int* b, int* c) {
    const int lane = threadIdx.x & 31;
    int base = 0;
    for (int b0 = 0; b0 < B; b0 += 32) {
        const int k = dl_chunks_of(cu, b0 + lane, B);
        int x = k;
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const int y = __shfl_up_sync(0xffffffffu, x, o);
            if (lane >= o) x += y;
        }
        const int total = __shfl_sync(0xffffffffu, x, 31);
        if (idx < base + total) {
            const int src = __ffs(__ballot_sync(0xffffffffu, base + x > idx)) - 1;
            *b = b0 + src;
            *c = idx - base - __shfl_sync(0xffffffffu, x - k, src);
            return true;
        }
        base += total;
    }
    return false;
}
__device__ __forceinline__ int dl_first_chunk(const int* cu, int b) {       // chunks of the requests before b; by whole warps
    int k = 0;
    for (int i = threadIdx.x & 31; i < b; i += 32) k += dl_chunks_of(cu, i, b);
#pragma unroll
    for (int o = 16; o > 0; o >>= 1) k += __shfl_xor_sync(0xffffffffu, k, o);
    return k;
}
// Buffers of a chunk and head (number i = chunk * H + head): Wt [D][64], Ut [P][64] (right sides solved, token index last),
// M [64][64], rows [3][64] (factor of q rows, factor of k rows, e^(L_64) in the first place), S0 [D][P].
#define DL_ROWS 3

// ------------------------------------------------------------------------------------------ (1) the chunks' own matrices
#define PREP_LDA (DC + 4)
template <typename TP>
__global__ void __launch_bounds__(256, 2)
delta_prep_kernel(const float* __restrict__ qkv, int C, const TP* __restrict__ proj, int ld, int a_col, int b_col,
                  const float* __restrict__ dt_bias, const float* __restrict__ A_log, float q_scale, float unit_eps,
                  const int* __restrict__ cu, int B, float* __restrict__ Wt, float* __restrict__ Ut, float* __restrict__ M,
                  float* __restrict__ rows, int H, int G, int D, int P) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float s_beta[DC], s_hi[DC], s_lo[DC], s_kn[DC], s_qn[DC];
    pdl_launch_dependents();
    pdl_wait();
    int b, c;
    if (!dl_find(cu, B, blockIdx.x, &b, &c)) return;
    const int h = blockIdx.y, g = h / (H / G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int row0 = cu[b] + c * DC, m = min(DC, cu[b + 1] - row0);
    const int LD = D + 4;
    float* K = sm;                                                // [64][D + 4]
    float* Q = K + DC * LD;
    float* At = Q + DC * LD;                                      // [64][68]: A transposed, token s first
    // a warp per row: the row's vectors made unit vectors on their way into shared memory
    for (int t = warp; t < DC; t += 8) {
        float4 q = make_float4(0.f, 0.f, 0.f, 0.f), k = q;
        if (t < m && 4 * lane < D) {
            const float* row = qkv + (size_t)(row0 + t) * C;
            q = ld4(row + (size_t)g * D + 4 * lane);
            k = ld4(row + (size_t)(G + g) * D + 4 * lane);
        }
        const float qn = q_scale / sqrtf(warp_sum(dot4(q, q)) + unit_eps), kn = 1.f / sqrtf(warp_sum(dot4(k, k)) + unit_eps);
        if (4 * lane < D) {
            st4(Q + t * LD + 4 * lane, make_float4(q.x * qn, q.y * qn, q.z * qn, q.w * qn));
            st4(K + t * LD + 4 * lane, make_float4(k.x * kn, k.y * kn, k.z * kn, k.w * kn));
        }
        if (lane == 0) { s_kn[t] = kn; s_qn[t] = qn; }
    }
    if (warp == 0) {                                              // two tokens a lane: beta, log decay, its running sum
        const float rate = expf(A_log[h]), bias = dt_bias[h];
        double l[2];
#pragma unroll
        for (int e = 0; e < 2; ++e) {
            const int t = 2 * lane + e;
            const TP* prow = proj + (size_t)(row0 + min(t, m - 1)) * ld;
            s_beta[t] = t < m ? dl_sigmoid(to_f32(prow[b_col + h])) : 0.f;
            l[e] = t < m ? (double)(-rate * dl_softplus(to_f32(prow[a_col + h]) + bias)) : 0.0;
        }
        double x = l[0] + l[1];
#pragma unroll
        for (int o = 1; o < 32; o <<= 1) {
            const double y = __shfl_up_sync(0xffffffffu, x, o);
            if (lane >= o) x += y;
        }
        const double first = x - l[1];
        s_hi[2 * lane] = (float)first;
        s_lo[2 * lane] = (float)(first - (double)(float)first);
        s_hi[2 * lane + 1] = (float)x;
        s_lo[2 * lane + 1] = (float)(x - (double)(float)x);
    }
    __syncthreads();
    const size_t ch = (size_t)blockIdx.x * H + h;
    if (tid < DC) {
        float* rw = rows + ch * DL_ROWS * DC;
        const bool on = tid < m;
        rw[tid] = on ? s_qn[tid] * expf(s_hi[tid] + s_lo[tid]) : 0.f;
        rw[DC + tid] = on ? s_kn[tid] * expf((s_hi[DC - 1] - s_hi[tid]) + (s_lo[DC - 1] - s_lo[tid])) : 0.f;
        if (tid == 0) rw[2 * DC] = expf(s_hi[DC - 1] + s_lo[DC - 1]);
    }
    // both products over D: token t = ty + 16 i against token s = tx + 16 j
    const int tx = tid & 15, ty = tid >> 4;
    float kk[4][4], qk[4][4];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int j = 0; j < 4; ++j) kk[i][j] = qk[i][j] = 0.f;
    for (int d = 0; d < D; d += 4) {
        float4 ks[4];
#pragma unroll
        for (int j = 0; j < 4; ++j) ks[j] = ld4(K + (tx + 16 * j) * LD + d);
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            const float4 kt = ld4(K + (ty + 16 * i) * LD + d), qt = ld4(Q + (ty + 16 * i) * LD + d);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                kk[i][j] += kt.x * ks[j].x; kk[i][j] += kt.y * ks[j].y; kk[i][j] += kt.z * ks[j].z; kk[i][j] += kt.w * ks[j].w;
                qk[i][j] += qt.x * ks[j].x; qk[i][j] += qt.y * ks[j].y; qk[i][j] += qt.z * ks[j].z; qk[i][j] += qt.w * ks[j].w;
            }
        }
    }
    float* Mo = M + ch * DC * DC;
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = ty + 16 * i;
#pragma unroll
        for (int j = 0; j < 4; ++j) {
            const int s = tx + 16 * j;
            const float f = s <= t ? expf((s_hi[t] - s_hi[s]) + (s_lo[t] - s_lo[s])) : 0.f;
            Mo[t * DC + s] = f * qk[i][j];
            At[s * PREP_LDA + t] = s < t ? s_beta[t] * f * kk[i][j] : 0.f;
        }
    }
    __syncthreads();
    // a thread per right side: (1 + A) x = [beta v | beta e^L k], forward, every x_s taken off all later tokens
    for (int col = tid; col < P + D; col += 256) {
        float x[DC];
        if (col < P) {
            const float* v = qkv + (size_t)row0 * C + (size_t)2 * G * D + (size_t)h * P + col;
#pragma unroll
            for (int t = 0; t < DC; ++t) x[t] = t < m ? s_beta[t] * v[(size_t)t * C] : 0.f;
        } else {
#pragma unroll
            for (int t = 0; t < DC; ++t) x[t] = s_beta[t] * (expf(s_hi[t] + s_lo[t]) * K[t * LD + col - P]);
        }
#pragma unroll
        for (int s = 0; s < DC - 1; ++s) {
            const float xs = x[s];
#pragma unroll
            for (int t = (s + 1) & ~3; t < DC; t += 4) {
                const float4 a = ld4(At + s * PREP_LDA + t);
                if (t > s) x[t] -= a.x * xs;
                if (t + 1 > s) x[t + 1] -= a.y * xs;
                if (t + 2 > s) x[t + 2] -= a.z * xs;
                x[t + 3] -= a.w * xs;
            }
        }
        float* dst = col < P ? Ut + (ch * P + col) * DC : Wt + (ch * D + col - P) * DC;
#pragma unroll
        for (int t = 0; t < DC; t += 4) st4(dst + t, make_float4(x[t], x[t + 1], x[t + 2], x[t + 3]));
    }
}

// ------------------------------------------------------------------------------------------ (2) from chunk to chunk
// A block owns CT value columns of one head of one request: the state's tile in registers (for its update) and in shared memory
// (for W S).  U goes to `U` [T][H P], the state at every chunk's start to S0.
template <int CT>
__global__ void __launch_bounds__(256)
delta_walk_kernel(const float* __restrict__ qkv, int C, const float* __restrict__ Wt, const float* __restrict__ Ut,
                  const float* __restrict__ rows, float* __restrict__ U, float* __restrict__ S0, float* __restrict__ state,
                  long long state_stride, const int* __restrict__ cu, const int* __restrict__ slots, int H, int G, int D, int P) {
    constexpr int CPT = CT / 8;                                   // phase 1: columns a thread (4 tokens each)
    constexpr int CG = CT / 4, DPT = DELTA_MAX * CG / 256;        // phase 2: groups of 4 columns, rows a thread
    extern __shared__ __align__(16) float sm[];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, b = blockIdx.y, p0 = blockIdx.z * CT;
    const int s0 = cu[b], n = cu[b + 1] - s0;
    if (n < DELTA_MIN_CHUNK) return;
    const int first = dl_first_chunk(cu, b), chunks = (n + DC - 1) / DC;
    const int g = h / (H / G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    const int stage = D * DC + DC * D + CT * DC + 2 * DC;         // W^T, k rows, U0^T, factors of the k rows and e^L
    float* Ss = sm + 2 * stage;                                   // [D][CT]
    float* red = Ss + D * CT;                                     // [64][CT]
    float* Us = red + DC * CT;                                    // [64][CT]: U times the k rows' factors
    auto fetch = [&](int c, int buf) {
        float* w = sm + buf * stage;
        float* k = w + D * DC;
        float* u = k + DC * D;
        float* f = u + CT * DC;
        const size_t ch = (size_t)(first + c) * H + h;
        for (int i = tid; i < D * DC / 4; i += 256) dl_copy16(w + 4 * i, Wt + ch * D * DC + 4 * i, true);
        const int per = D / 4, m = min(DC, n - c * DC);
        for (int i = tid; i < DC * per; i += 256) {
            const int t = i / per, d = 4 * (i - t * per);
            const bool ok = t < m;
            dl_copy16(k + t * D + d, ok ? qkv + (size_t)(s0 + c * DC + t) * C + (size_t)(G + g) * D + d : qkv, ok);
        }
        for (int i = tid; i < CT * DC / 4; i += 256) {
            const bool ok = p0 + i / (DC / 4) < P;
            dl_copy16(u + 4 * i, ok ? Ut + (ch * P + p0) * DC + 4 * i : Ut, ok);
        }
        if (tid < 2 * DC / 4) dl_copy16(f + 4 * tid, rows + ch * DL_ROWS * DC + DC + 4 * tid, true);
    };
    // phase 2 ownership: rows d0 .. d0 + DPT - 1, columns 4 cg ..
    const int cg2 = lane % 4 + 4 * (CG == 8 ? warp & 1 : 0), d0 = DPT * ((lane >> 2) + 8 * (CG == 8 ? warp >> 1 : warp));
    float* gs = state + (long long)slots[b] * state_stride + (size_t)h * D * P + p0 + 4 * cg2;
    const bool own_cols = p0 + 4 * cg2 < P;
    float4 sr[DPT];
#pragma unroll
    for (int i = 0; i < DPT; ++i) {
        sr[i] = (own_cols && d0 + i < D) ? ld4(gs + (size_t)(d0 + i) * P) : make_float4(0.f, 0.f, 0.f, 0.f);
        if (d0 + i < D) st4(Ss + (d0 + i) * CT + 4 * cg2, sr[i]);
    }
    // phase 1 ownership: a half of the rows d, tokens t0 .. t0 + 3, columns c1 .. c1 + CPT - 1
    const int half = warp >> 2, w4 = warp & 3;
    const int t0 = 4 * ((w4 & 1) * 8 + (lane & 7)), c1 = CPT * ((w4 >> 1) * 4 + (lane >> 3));
    const int dlo = half ? D / 2 : 0, dhi = half ? D : D / 2;
    fetch(0, 0);
    dl_commit();
    for (int c = 0; c < chunks; ++c) {
        dl_wait<0>();
        __syncthreads();
        if (c + 1 < chunks) { fetch(c + 1, (c + 1) & 1); dl_commit(); }
        const float* w = sm + (c & 1) * stage;
        const float* k = w + D * DC;
        const float* u = k + DC * D;
        const float* f = u + CT * DC;
        if (own_cols) {
            float* so = S0 + (((size_t)(first + c) * H + h) * D) * P + p0 + 4 * cg2;
#pragma unroll
            for (int i = 0; i < DPT; ++i)
                if (d0 + i < D) st4(so + (size_t)(d0 + i) * P, sr[i]);
        }
        float acc[CPT][4];
#pragma unroll
        for (int j = 0; j < CPT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll 8
        for (int d = dlo; d < dhi; ++d) {
            const float4 a = ld4(w + d * DC + t0);
            float s[CPT];
            if constexpr (CPT == 4) {
                const float4 q = ld4(Ss + d * CT + c1);
                s[0] = q.x; s[1] = q.y; s[2] = q.z; s[3] = q.w;
            } else {
                const float2 q = *reinterpret_cast<const float2*>(Ss + d * CT + c1);
                s[0] = q.x; s[1] = q.y;
            }
#pragma unroll
            for (int j = 0; j < CPT; ++j) {
                acc[j][0] += a.x * s[j]; acc[j][1] += a.y * s[j]; acc[j][2] += a.z * s[j]; acc[j][3] += a.w * s[j];
            }
        }
        if (half) {
#pragma unroll
            for (int e = 0; e < 4; ++e)
#pragma unroll
                for (int j = 0; j < CPT; ++j) red[(t0 + e) * CT + c1 + j] = acc[j][e];
        }
        __syncthreads();
        if (!half) {
            const int m = min(DC, n - c * DC);
#pragma unroll
            for (int e = 0; e < 4; ++e) {
                const int t = t0 + e;
                float v[CPT];
#pragma unroll
                for (int j = 0; j < CPT; ++j) {
                    v[j] = u[(c1 + j) * DC + t] - (acc[j][e] + red[t * CT + c1 + j]);
                    Us[t * CT + c1 + j] = v[j] * f[t];
                }
                if (t < m && p0 + c1 < P) {
                    float* dst = U + (size_t)(s0 + c * DC + t) * H * P + (size_t)h * P + p0 + c1;
                    if constexpr (CPT == 4) st4(dst, make_float4(v[0], v[1], v[2], v[3]));
                    else *reinterpret_cast<float2*>(dst) = make_float2(v[0], v[1]);
                }
            }
        }
        __syncthreads();
        const float keep = f[DC];
#pragma unroll
        for (int i = 0; i < DPT; ++i) { sr[i].x *= keep; sr[i].y *= keep; sr[i].z *= keep; sr[i].w *= keep; }
        if (d0 < D) {
#pragma unroll 8
            for (int t = 0; t < DC; ++t) {
                const float4 v = ld4(Us + t * CT + 4 * cg2);
                float kd[DPT];
                if constexpr (DPT == 4) {
                    const float4 q = ld4(k + t * D + d0);
                    kd[0] = q.x; kd[1] = q.y; kd[2] = q.z; kd[3] = q.w;
                } else {
                    const float2 q = *reinterpret_cast<const float2*>(k + t * D + d0);
                    kd[0] = q.x; kd[1] = q.y;
                }
#pragma unroll
                for (int i = 0; i < DPT; ++i) {
                    sr[i].x += kd[i] * v.x; sr[i].y += kd[i] * v.y; sr[i].z += kd[i] * v.z; sr[i].w += kd[i] * v.w;
                }
            }
#pragma unroll
            for (int i = 0; i < DPT; ++i)
                if (d0 + i < D) st4(Ss + (d0 + i) * CT + 4 * cg2, sr[i]);
        }
    }
    if (own_cols) {
#pragma unroll
        for (int i = 0; i < DPT; ++i)
            if (d0 + i < D) st4(gs + (size_t)(d0 + i) * P, sr[i]);
    }
}

// ------------------------------------------------------------------------------------------ (3) the chunks' outputs
#define OUT_BK 32
template <typename TP, int NC>
__global__ void __launch_bounds__(256, 2)
delta_out_kernel(const float* __restrict__ qkv, int C, const TP* __restrict__ proj, int ld, int gate_col, const float* __restrict__ M,
                 const float* __restrict__ rows, const float* __restrict__ U, const float* __restrict__ S0,
                 const float* __restrict__ norm, float eps, const int* __restrict__ cu, int B, TP* __restrict__ out, int H, int G,
                 int D, int P) {
    constexpr int LDP = 64 * NC;                                  // columns of a staged row
    extern __shared__ __align__(16) float sm[];
    pdl_launch_dependents();
    pdl_wait();
    int b, c;
    if (!dl_find(cu, B, blockIdx.x, &b, &c)) return;
    const int h = blockIdx.y, g = h / (H / G), tid = threadIdx.x;
    const int row0 = cu[b] + c * DC, m = min(DC, cu[b + 1] - row0);
    const size_t ch = (size_t)blockIdx.x * H + h;
    const int LD = D + 4, LM = DC + 4;
    float* Q = sm;                                                // [64][D + 4]
    float* Ms = Q + DC * LD;                                      // [64][68]
    float* Bs = Ms + DC * LM;                                     // two stages of [32][LDP]
    const int nS = (D + OUT_BK - 1) / OUT_BK, tiles = nS + DC / OUT_BK;
    auto fetch = [&](int tile, int buf) {
        float* dst = Bs + buf * OUT_BK * LDP;
        const bool from_state = tile < nS;
        const int r0 = (from_state ? tile : tile - nS) * OUT_BK;
        const float* src = from_state ? S0 + ch * D * P : U + (size_t)row0 * H * P + (size_t)h * P;
        const size_t stride = from_state ? P : (size_t)H * P;
        const int last = from_state ? D : m;
        for (int i = tid; i < OUT_BK * LDP / 4; i += 256) {
            const int r = i / (LDP / 4), col = 4 * (i - r * (LDP / 4));
            const bool ok = r0 + r < last && col < P;
            dl_copy16(dst + r * LDP + col, ok ? src + (size_t)(r0 + r) * stride + col : src, ok);
        }
    };
    {
        const int per = D / 4;
        for (int i = tid; i < DC * per; i += 256) {
            const int t = i / per, d = 4 * (i - t * per);
            const bool ok = t < m;
            dl_copy16(Q + t * LD + d, ok ? qkv + (size_t)(row0 + t) * C + (size_t)g * D + d : qkv, ok);
        }
        for (int i = tid; i < DC * DC / 4; i += 256) {
            const int t = i / (DC / 4), s = 4 * (i - t * (DC / 4));
            dl_copy16(Ms + t * LM + s, M + ch * DC * DC + 4 * i, true);
        }
    }
    fetch(0, 0);
    dl_commit();
    const int tx = tid & 15, ty = tid >> 4;                       // tokens 4 ty + i, columns 4 tx + 64 e
    float4 acc[4][NC];
#pragma unroll
    for (int i = 0; i < 4; ++i)
#pragma unroll
        for (int e = 0; e < NC; ++e) acc[i][e] = make_float4(0.f, 0.f, 0.f, 0.f);
    const float* rw = rows + ch * DL_ROWS * DC;
    for (int tile = 0; tile < tiles; ++tile) {
        dl_wait<0>();
        __syncthreads();
        if (tile + 1 < tiles) { fetch(tile + 1, (tile + 1) & 1); dl_commit(); }
        if (tile == nS) {                                         // what the state gives is complete: the rows' own factors
#pragma unroll
            for (int i = 0; i < 4; ++i) {
                const float f = rw[4 * ty + i];
#pragma unroll
                for (int e = 0; e < NC; ++e) { acc[i][e].x *= f; acc[i][e].y *= f; acc[i][e].z *= f; acc[i][e].w *= f; }
            }
        }
        const bool from_state = tile < nS;
        const float* A = from_state ? Q + tile * OUT_BK : Ms + (tile - nS) * OUT_BK;
        const int lda = from_state ? LD : LM;
        const int depth = from_state ? min(OUT_BK, D - tile * OUT_BK) : OUT_BK;
        const float* Bt = Bs + (tile & 1) * OUT_BK * LDP + 4 * tx;
        for (int k = 0; k < depth; k += 4) {
            float4 a[4];
#pragma unroll
            for (int i = 0; i < 4; ++i) a[i] = ld4(A + (4 * ty + i) * lda + k);
#pragma unroll
            for (int kk = 0; kk < 4; ++kk) {
                float4 v[NC];
#pragma unroll
                for (int e = 0; e < NC; ++e) v[e] = ld4(Bt + (k + kk) * LDP + 64 * e);
#pragma unroll
                for (int i = 0; i < 4; ++i) {
                    const float x = kk == 0 ? a[i].x : (kk == 1 ? a[i].y : (kk == 2 ? a[i].z : a[i].w));
#pragma unroll
                    for (int e = 0; e < NC; ++e) {
                        acc[i][e].x += x * v[e].x; acc[i][e].y += x * v[e].y; acc[i][e].z += x * v[e].z; acc[i][e].w += x * v[e].w;
                    }
                }
            }
        }
    }
#pragma unroll
    for (int i = 0; i < 4; ++i) {
        const int t = 4 * ty + i;
        float ss = 0.f;
#pragma unroll
        for (int e = 0; e < NC; ++e) ss += dot4(acc[i][e], acc[i][e]);     // (columns behind P are zero)
#pragma unroll
        for (int o = 8; o > 0; o >>= 1) ss += __shfl_xor_sync(0xffffffffu, ss, o);
        const float inv = 1.f / sqrtf(ss / (float)P + eps);
        if (t >= m) continue;
#pragma unroll
        for (int e = 0; e < NC; ++e) {
            const int col = 4 * tx + 64 * e;
            if (col >= P) continue;
            const float4 nw = ld4(norm + col), z = Quad<TP>::load(proj + (size_t)(row0 + t) * ld + gate_col + (size_t)h * P + col);
            Quad<TP>::store(out + (size_t)(row0 + t) * H * P + (size_t)h * P + col,
                            make_float4(acc[i][e].x * inv * nw.x * dl_silu(z.x), acc[i][e].y * inv * nw.y * dl_silu(z.y),
                                        acc[i][e].z * inv * nw.z * dl_silu(z.z), acc[i][e].w * inv * nw.w * dl_silu(z.w)));
        }
    }
}

extern "C" int vl_delta_min_chunk() { return DELTA_MIN_CHUNK; }
// Floats of the scratch for a launch of up to `chunks` chunks: W^T, U0^T, M, row factors, chunk states (U has its own [T, H P]).
extern "C" long long vl_delta_chunk_floats(int chunks, int H, int D, int P) {
    return (long long)chunks * H * ((long long)D * DC + (long long)P * DC + DC * DC + DL_ROWS * DC + (long long)D * P);
}

template <typename K>
static int delta_smem(K kernel, size_t bytes) {
    return (int)cudaFuncSetAttribute(kernel, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)bytes);
}
template <int CT>
static int launch_walk(const float* qkv, int C, const float* Wt, const float* Ut, const float* rows, float* U, float* S0, float* state,
                       long long state_stride, const int* cu, const int* slots, int B, int H, int G, int D, int P, cudaStream_t s) {
    const size_t smem = sizeof(float) * ((size_t)2 * (2 * D * DC + CT * DC + 2 * DC) + (size_t)D * CT + 2 * DC * CT);
    const int rc = delta_smem(delta_walk_kernel<CT>, smem);
    if (rc) return rc;
    return vl_launch(delta_walk_kernel<CT>, dim3(H, B, (P + CT - 1) / CT), dim3(256), smem, s, qkv, C, Wt, Ut, rows, U, S0, state, state_stride,
                     cu, slots, H, G, D, P);
}
template <typename TP>
static int launch_chunks(const float* qkv, int C, const TP* proj, int ld, int a_col, int b_col, int gate_col, const float* dt_bias,
                         const float* A_log, float q_scale, float unit_eps, const float* norm, float eps, float* state,
                         long long state_stride, const int* cu, const int* slots, int B, int chunks, float* scratch, float* U, TP* out,
                         int H, int G, int D, int P, int sms, cudaStream_t s) {
    const size_t n = (size_t)chunks * H;
    float* Wt = scratch;
    float* Ut = Wt + n * D * DC;
    float* M = Ut + n * P * DC;
    float* rows = M + n * DC * DC;
    float* S0 = rows + n * DL_ROWS * DC;
    size_t smem = sizeof(float) * ((size_t)2 * DC * (D + 4) + DC * PREP_LDA);
    int rc = delta_smem(delta_prep_kernel<TP>, smem);
    if (rc) return rc;
    rc = vl_launch(delta_prep_kernel<TP>, dim3(chunks, H), dim3(256), smem, s, qkv, C, proj, ld, a_col, b_col, dt_bias, A_log, q_scale,
                   unit_eps, cu, B, Wt, Ut, M, rows, H, G, D, P);
    if (rc) return rc;
    // narrow tiles of columns while they leave an SM to every block
    if ((long long)H * B * ((P + 15) / 16) <= sms)
        rc = launch_walk<16>(qkv, C, Wt, Ut, rows, U, S0, state, state_stride, cu, slots, B, H, G, D, P, s);
    else
        rc = launch_walk<32>(qkv, C, Wt, Ut, rows, U, S0, state, state_stride, cu, slots, B, H, G, D, P, s);
    if (rc) return rc;
#define DELTA_OUT(NC)                                                                                                               \
    do {                                                                                                                            \
        smem = sizeof(float) * ((size_t)DC * (D + 4) + DC * (DC + 4) + 2 * OUT_BK * 64 * NC);                                       \
        rc = delta_smem(delta_out_kernel<TP, NC>, smem);                                                                            \
        if (rc) return rc;                                                                                                          \
        return vl_launch(delta_out_kernel<TP, NC>, dim3(chunks, H), dim3(256), smem, s, qkv, C, proj, ld, gate_col, M, rows, U, S0, \
                         norm, eps, cu, B, out, H, G, D, P);                                                                        \
    } while (0)
    if (P <= 64) DELTA_OUT(1);
    DELTA_OUT(2);
#undef DELTA_OUT
}

// `chunks`: a bound on the chunks of the step (its tokens / 64 plus its requests); scratch: vl_delta_chunk_floats(chunks) floats;
// U float32 [T, H P].  Requests of fewer than DELTA_MIN_CHUNK tokens are passed over (vl_delta_step serves them).
extern "C" int vl_delta_chunks(const float* qkv, int C, const void* proj, int dtype, int ld, int a_col, int b_col, int gate_col,
                               const float* dt_bias, const float* A_log, float q_scale, float unit_eps, const float* norm, float eps,
                               float* state, long long state_stride, const int* cu, const int* slots, int B, int chunks, float* scratch,
                               float* U, void* out, int H, int G, int D, int P, int sms, void* stream) {
    if (B <= 0 || chunks <= 0) return VL_OK;
    if (!delta_sizes_ok(H, G, D, P, C) || B > 65535 || H > 65535) return VL_ERR_UNSUPPORTED;
    if (ld % 4 || gate_col % 4 || state_stride % 4 ||
        (((uintptr_t)qkv | (uintptr_t)proj | (uintptr_t)state | (uintptr_t)out | (uintptr_t)norm | (uintptr_t)scratch | (uintptr_t)U) & 15))
        return VL_ERR_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == VL_F32)
        return launch_chunks<float>(qkv, C, (const float*)proj, ld, a_col, b_col, gate_col, dt_bias, A_log, q_scale, unit_eps, norm, eps,
                                    state, state_stride, cu, slots, B, chunks, scratch, U, (float*)out, H, G, D, P, sms, s);
    if (dtype == VL_BF16)
        return launch_chunks<bf16>(qkv, C, (const bf16*)proj, ld, a_col, b_col, gate_col, dt_bias, A_log, q_scale, unit_eps, norm, eps,
                                   state, state_stride, cu, slots, B, chunks, scratch, U, (bf16*)out, H, G, D, P, sms, s);
    return VL_ERR_UNSUPPORTED;
}
