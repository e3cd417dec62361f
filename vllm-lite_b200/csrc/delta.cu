// The gated delta rule with ONE decay per head, for states of up to 128 x 128 numbers a head:
//     S <- g S;  u = beta (v - S^T k);  S <- S + k u^T;  o = S^T q         then   out = rms_head(o) * norm * silu(gate)
// over the tokens that a step brings for every request (rows cu[b] .. cu[b+1]-1), from the state in the request's slot.
// q, k, v are columns of `qkv` (float32, what the short convolution leaves: q heads | k heads | v heads), the raw decay and
// the raw beta columns of the stacked product's rows, the gate another block of columns there.  k and q are made unit
// vectors (q times q_scale), g = exp(-exp(A_log) softplus(a + dt_bias)), beta = sigmoid(b).  Everything is float32: no product
// here runs in fewer bits.  A head's state lies row by row, [D][P].
//
//   vl_delta_step    portions of fewer than DELTA_MIN_CHUNK tokens (decoding): a block holds the whole state of a (head, request) in
//                    registers while its tokens pass; states come and go by bulk copies through a ring in shared memory.
//                    One pass over the state and one sum across the block a token: with w = S^T k and r = S^T q of
//                    the old state, u = beta (v - g w) and o = g r + (k.q) u.
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
#include "tc5.cuh"

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
__device__ __forceinline__ void dl_copy8(void* smem, const void* gmem, bool valid) {
    const unsigned dst = (unsigned)__cvta_generic_to_shared(smem);
    const int bytes = valid ? 8 : 0;
    asm volatile("cp.async.ca.shared.global [%0], [%1], 8, %2;" ::"r"(dst), "l"(gmem), "r"(bytes) : "memory");
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
// A block works off every gridDim-th (request, head); the states of the heads pass through a ring of STEP_STAGES places in shared
// memory: the bulk copy of the next one is on its way in, and the one before on its way back, while a state is worked on.
#define STEP_STAGES 3
__device__ __forceinline__ void dl_bulk_load(void* smem, const void* gmem, unsigned bytes, unsigned long long* bar) {
    asm volatile("cp.async.bulk.shared::cluster.global.mbarrier::complete_tx::bytes [%0], [%1], %2, [%3];"
                 ::"r"(tc5::smem_u32(smem)), "l"(gmem), "r"(bytes), "r"(tc5::smem_u32(bar)) : "memory");
}
__device__ __forceinline__ void dl_bulk_store(void* gmem, const void* smem, unsigned bytes) {
    asm volatile("cp.async.bulk.global.shared::cta.bulk_group [%0], [%1], %2;" ::"l"(gmem), "r"(tc5::smem_u32(smem)), "r"(bytes) : "memory");
    asm volatile("cp.async.bulk.commit_group;" ::: "memory");
}
template <typename TP>
__global__ void __launch_bounds__(512, 1)
delta_step_kernel(const float* __restrict__ qkv, int C, const TP* __restrict__ proj, int ld, int a_col, int b_col, int gate_col,
                  const float* __restrict__ dt_bias, const float* __restrict__ A_log, float q_scale, float unit_eps,
                  const float* __restrict__ norm, float eps, float* __restrict__ state, long long state_stride,
                  const int* __restrict__ cu, const int* __restrict__ slots, TP* __restrict__ out, int H, int G, int D, int P,
                  int longest, int LU, int UG, int WR, int items, unsigned* err) {
    extern __shared__ __align__(128) float ring[];                 // [STEP_STAGES][D][P]
    __shared__ __align__(16) float sq[DELTA_MAX], sk[DELTA_MAX], su[DELTA_MAX], part[2][4][DELTA_MAX];
    __shared__ float s_g, s_beta, s_qk;
    __shared__ unsigned long long full[STEP_STAGES];
    const int tid = threadIdx.x, warp = tid >> 5, lane = tid & 31;
    if (tid == 0) {
        for (int i = 0; i < STEP_STAGES; ++i) tc5::mbar_init(&full[i], 1);
        tc5::mbar_fence_init();
    }
    pdl_launch_dependents();
    pdl_wait();
    __syncthreads();
    const int U = P >> 2, RG = WR * (32 / LU), grid = gridDim.x;
    const int unit = (warp % UG) * LU + lane % LU, wr = warp / UG, rg = wr * (32 / LU) + lane / LU;
    const bool live = unit < U;
    const bool lead = warp == (int)(blockDim.x >> 5) - 1 && lane == 0;       // issues the copies, makes the head's two numbers
    const unsigned bytes = (unsigned)(sizeof(float) * D * P);
    auto next = [&](int it) {                                     // the first of this block's items from `it` on that has work here
        while (it < items) {
            const int b = it / H, n = cu[b + 1] - cu[b];
            if (n > 0 && n <= longest) break;
            it += grid;
        }
        return it;
    };
    auto place = [&](int it) { const int b = it / H; return state + (long long)slots[b] * state_stride + (size_t)(it - b * H) * D * P; };
    auto load = [&](int it, int stage) {
        tc5::mbar_arrive_expect_tx(&full[stage], bytes);
        dl_bulk_load(ring + (size_t)stage * D * P, place(it), bytes, &full[stage]);
    };
    // what the first token of an item needs beside the state is asked for while the item before is worked on
    float4 q4, k4, v4, z4;
    float ra = 0.f, rb = 0.f;
    auto ask = [&](int it, int t) {
        const int b = it / H, h = it - b * H, g = h / (H / G);
        const float* row = qkv + (size_t)(cu[b] + t) * C;
        const TP* prow = proj + (size_t)(cu[b] + t) * ld;
        if (warp == 0) {
            q4 = k4 = v4 = z4 = make_float4(0.f, 0.f, 0.f, 0.f);
            if (4 * lane < D) { q4 = ld4(row + (size_t)g * D + 4 * lane); k4 = ld4(row + (size_t)(G + g) * D + 4 * lane); }
            if (lane < U) {
                v4 = ld4(row + (size_t)2 * G * D + (size_t)h * P + 4 * lane);
                z4 = Quad<TP>::load(prow + gate_col + (size_t)h * P + 4 * lane);
            }
        }
        if (lead) { ra = to_f32(prow[a_col + h]); rb = to_f32(prow[b_col + h]); }
    };
    int cur = next(blockIdx.x), nxt = next(cur + grid);
    if (lead) {
        if (cur < items) load(cur, 0);
        if (nxt < items) load(nxt, 1);
    }
    if (cur < items) ask(cur, 0);
    bool ok = true;
    int j = 0;
    for (; cur < items; ++j) {
        const int third = next(nxt + grid), stage = j % STEP_STAGES;
        const int b = cur / H, h = cur - b * H, s0 = cu[b], n = cu[b + 1] - s0;
        float* S = ring + (size_t)stage * D * P + 4 * unit;
        float4 s[STEP_ROWS];
        for (int t = 0; t < n; ++t) {
            const float4 v = v4, z = z4;
            if (warp == 0) {                                      // unit vectors and their product
                float4 q = q4, k = k4;
                const float qn = q_scale / sqrtf(warp_sum(dot4(q, q)) + unit_eps), kn = 1.f / sqrtf(warp_sum(dot4(k, k)) + unit_eps);
                q.x *= qn; q.y *= qn; q.z *= qn; q.w *= qn;
                k.x *= kn; k.y *= kn; k.z *= kn; k.w *= kn;
                if (4 * lane < D) { st4(sq + 4 * lane, q); st4(sk + 4 * lane, k); }
                const float qk = warp_sum(dot4(q, k));
                if (lane == 0) s_qk = qk;
            }
            if (lead) {
                s_g = expf(-expf(A_log[h]) * dl_softplus(ra + dt_bias[h]));
                s_beta = dl_sigmoid(rb);
            }
            if (t == 0) ok = tc5::mbar_wait_bounded(&full[stage], (unsigned)((j / STEP_STAGES) & 1));
            if (!__syncthreads_and(ok)) { ok = false; break; }
            if (t + 1 < n) ask(cur, t + 1);
            else if (nxt < items) ask(nxt, 0);
            if (t == 0) {
#pragma unroll
                for (int i = 0; i < STEP_ROWS; ++i) {
                    const int r = rg + RG * i;
                    s[i] = (live && r < D) ? ld4(S + r * P) : make_float4(0.f, 0.f, 0.f, 0.f);
                }
            }
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
            for (int o = LU; o < 32; o <<= 1) {                   // the warp's rows of a unit
                w.x += __shfl_xor_sync(0xffffffffu, w.x, o); w.y += __shfl_xor_sync(0xffffffffu, w.y, o);
                w.z += __shfl_xor_sync(0xffffffffu, w.z, o); w.w += __shfl_xor_sync(0xffffffffu, w.w, o);
                r4.x += __shfl_xor_sync(0xffffffffu, r4.x, o); r4.y += __shfl_xor_sync(0xffffffffu, r4.y, o);
                r4.z += __shfl_xor_sync(0xffffffffu, r4.z, o); r4.w += __shfl_xor_sync(0xffffffffu, r4.w, o);
            }
            if (live && lane < LU) {
                st4(&part[0][wr][4 * unit], w);
                st4(&part[1][wr][4 * unit], r4);
            }
            if (t == 0 && lead && third < items) {                // the place of the item before this one, once it has been read out
                asm volatile("cp.async.bulk.wait_group.read 0;" ::: "memory");
                load(third, (j + 2) % STEP_STAGES);
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
                if (live && r < D) {
                    const float kr = sk[r];
                    s[i].x = gt * s[i].x + kr * u.x; s[i].y = gt * s[i].y + kr * u.y;
                    s[i].z = gt * s[i].z + kr * u.z; s[i].w = gt * s[i].w + kr * u.w;
                    if (t + 1 == n) st4(S + r * P, s[i]);
                }
            }
            if (t + 1 == n) tc5::fence_proxy_async_smem();
            __syncthreads();                                      // the next token's unit vectors take sq and sk; the state is complete
        }
        if (!ok) break;
        if (lead) dl_bulk_store(place(cur), ring + (size_t)stage * D * P, bytes);
        cur = nxt;
        nxt = third;
    }
    if (lead) {
        if (!ok) {                                                // what is still on its way in must land before the block leaves
            if (err) atomicOr(err, VL_DEV_WAIT_EXPIRED | VL_DEV_IN_DELTA);
            tc5::mbar_wait_bounded(&full[j % STEP_STAGES], (unsigned)((j / STEP_STAGES) & 1));
            if (nxt < items) tc5::mbar_wait_bounded(&full[(j + 1) % STEP_STAGES], (unsigned)(((j + 1) / STEP_STAGES) & 1));
        }
        asm volatile("cp.async.bulk.wait_group 0;" ::: "memory");
    }
}

extern "C" int vl_delta_step(const float* qkv, int C, const void* proj, int dtype, int ld, int a_col, int b_col, int gate_col,
                             const float* dt_bias, const float* A_log, float q_scale, float unit_eps, const float* norm, float eps,
                             float* state, long long state_stride, const int* cu, const int* slots, int B, void* out, int H, int G,
                             int D, int P, int longest, int sms, unsigned* err, void* stream) {
    if (B <= 0) return VL_OK;
    if (!delta_sizes_ok(H, G, D, P, C)) return VL_ERR_UNSUPPORTED;
    if (ld % 4 || gate_col % 4 || state_stride % 4 || sms <= 0 || longest <= 0 ||
        (((uintptr_t)qkv | (uintptr_t)proj | (uintptr_t)state | (uintptr_t)out | (uintptr_t)norm) & 15))
        return VL_ERR_ARGUMENT;
    const StepShape sh = step_shape(D, P / 4);                    // (at most 16 warps, four rows of them)
    const size_t smem = sizeof(float) * (size_t)STEP_STAGES * D * P;
    const long long items = (long long)B * H, per_sm = (size_t)200 * 1024 / smem < 1 ? 1 : (200 * 1024 / smem > 4 ? 4 : 200 * 1024 / smem);
    if (items > 0x7fffffff) return VL_ERR_UNSUPPORTED;
    const long long most = (long long)sms * per_sm;
    cudaStream_t s = (cudaStream_t)stream;
#define DELTA_STEP(TP)                                                                                                              \
    do {                                                                                                                            \
        const cudaError_t e = cudaFuncSetAttribute(delta_step_kernel<TP>, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);  \
        if (e != cudaSuccess) return (int)e;                                                                                        \
        return vl_launch(delta_step_kernel<TP>, dim3((unsigned)(items < most ? items : most)), dim3(32 * sh.UG * sh.WR), smem, s, qkv, C, \
                         (const TP*)proj, ld, a_col, b_col, gate_col, dt_bias, A_log, q_scale, unit_eps, norm, eps, state, state_stride,  \
                         cu, slots, (TP*)out, H, G, D, P, longest, sh.LU, sh.UG, sh.WR, (int)items, err);                           \
    } while (0)
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

__device__ __forceinline__ float2 dl_load2(const float* p) { return *reinterpret_cast<const float2*>(p); }
__device__ __forceinline__ float2 dl_load2(const bf16* p) { return __bfloat1622float2(*reinterpret_cast<const __nv_bfloat162*>(p)); }
__device__ __forceinline__ void dl_store2(float* p, float a, float b) { *reinterpret_cast<float2*>(p) = make_float2(a, b); }
__device__ __forceinline__ void dl_store2(bf16* p, float a, float b) { *reinterpret_cast<__nv_bfloat162*>(p) = __floats2bfloat162_rn(a, b); }

// beta and the running sum of the log decays (as two floats) of a chunk's tokens, two a lane; tokens behind the portion: beta 0,
// no decay.  One warp.
struct RawDecays { float a[2], b[2], rate, bias; };
template <typename TP>
__device__ __forceinline__ RawDecays dl_load_decays(const TP* __restrict__ proj, int ld, int a_at, int b_at, int row0, int m,
                                                    const float* A_log, const float* dt_bias) {
    RawDecays r;
#pragma unroll
    for (int e = 0; e < 2; ++e) {                                 // (behind the portion: a number that is not used)
        const TP* prow = proj + (size_t)(row0 + min(2 * (int)(threadIdx.x & 31) + e, m - 1)) * ld;
        r.a[e] = to_f32(prow[a_at]);
        r.b[e] = to_f32(prow[b_at]);
    }
    r.rate = *A_log;
    r.bias = *dt_bias;
    return r;
}
__device__ __forceinline__ void dl_decays(const RawDecays& r, int m, float* beta, float* hi, float* lo) {
    const int lane = threadIdx.x & 31;
    const float rate = expf(r.rate);
    double l[2];
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const int t = 2 * lane + e;
        beta[t] = t < m ? dl_sigmoid(r.b[e]) : 0.f;
        l[e] = t < m ? (double)(-rate * dl_softplus(r.a[e] + r.bias)) : 0.0;
    }
    double x = l[0] + l[1];
#pragma unroll
    for (int o = 1; o < 32; o <<= 1) {
        const double y = __shfl_up_sync(0xffffffffu, x, o);
        if (lane >= o) x += y;
    }
    const double first = x - l[1];
    hi[2 * lane] = (float)first;
    lo[2 * lane] = (float)(first - (double)(float)first);
    hi[2 * lane + 1] = (float)x;
    lo[2 * lane + 1] = (float)(x - (double)(float)x);
}
// what the later launches multiply token t's rows by: q by its norm's inverse and e^(L_t), k by its norm's and e^(L_64 - L_t)
__device__ __forceinline__ void dl_row_factors(float* rw, int t, int m, const float* qn, const float* kn, const float* hi, const float* lo) {
    const bool on = t < m;
    rw[t] = on ? qn[t] * expf(hi[t] + lo[t]) : 0.f;
    rw[DC + t] = on ? kn[t] * expf((hi[DC - 1] - hi[t]) + (lo[DC - 1] - lo[t])) : 0.f;
    if (t == 0) rw[2 * DC] = expf(hi[DC - 1] + lo[DC - 1]);
}

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
    if (warp == 0) dl_decays(dl_load_decays(proj, ld, a_col + h, b_col + h, row0, m, A_log + h, dt_bias + h), m, s_beta, s_hi, s_lo);
    __syncthreads();
    const size_t ch = (size_t)blockIdx.x * H + h;
    if (tid < DC) dl_row_factors(rows + ch * DL_ROWS * DC, tid, m, s_qn, s_kn, s_hi, s_lo);
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

// ------------------------------------------------------------------------------------------ the chunks on the tensor cores
// In bfloat16 steps the products inside the chunks run on the tensor cores without losing float32's bits: a float32 number is
// the sum of three bfloat16 numbers (8 + 8 + 8 bits: hi = bf16(x), mid = bf16(x - hi), lo = bf16(x - hi - mid)), the products of
// bfloat16 numbers are exact in float32, and of the nine products of parts the six down to 2^-16 of the largest are added, in
// float32, the small ones first; what is left out lies below 2^-24 of a product (Henry, Tang, Heinecke, "Leveraging the
// bfloat16 Artificial Intelligence Datatype For Higher-Precision Computations").  Operands stay float32 in memory and are split in
// registers as fragments of mma.sync m16n8k16.  Same three launches, the same buffers (W and U0 row by row, [64][D], [64][P]).
struct FragA { unsigned h[4], m[4], l[4]; };
struct FragB { unsigned h[2], m[2], l[2]; };
__device__ __forceinline__ void split2(float x, float y, unsigned& h, unsigned& m, unsigned& l) {
    auto pack = [](float a, float b) {
        __nv_bfloat162 v = __floats2bfloat162_rn(a, b);
        return *reinterpret_cast<unsigned*>(&v);
    };
    h = pack(x, y);
    x -= __uint_as_float(h << 16);
    y -= __uint_as_float(h & 0xffff0000u);
    m = pack(x, y);
    l = pack(x - __uint_as_float(m << 16), y - __uint_as_float(m & 0xffff0000u));
}
// rows r, r + 8 and columns k, k + 1, k + 8, k + 9 (r, k: this lane's own) of a matrix stored row by row / column by column
__device__ __forceinline__ void frag_a_rows(FragA& f, const float* p, int ld, int r, int k) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const float2 v = *reinterpret_cast<const float2*>(p + (r + 8 * (e & 1)) * ld + k + 8 * (e >> 1));
        split2(v.x, v.y, f.h[e], f.m[e], f.l[e]);
    }
}
__device__ __forceinline__ void frag_a_cols(FragA& f, const float* p, int ld, int r, int k) {
#pragma unroll
    for (int e = 0; e < 4; ++e) {
        const float* q = p + (k + 8 * (e >> 1)) * ld + r + 8 * (e & 1);
        split2(q[0], q[ld], f.h[e], f.m[e], f.l[e]);
    }
}
// column n, rows k, k + 1, k + 8, k + 9 of B: stored with k along a row ([n][k]) / with n along a row ([k][n])
__device__ __forceinline__ void frag_b_nk(FragB& f, const float* p, int ld, int n, int k) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const float2 v = *reinterpret_cast<const float2*>(p + n * ld + k + 8 * e);
        split2(v.x, v.y, f.h[e], f.m[e], f.l[e]);
    }
}
__device__ __forceinline__ void frag_b_kn(FragB& f, const float* p, int ld, int n, int k) {
#pragma unroll
    for (int e = 0; e < 2; ++e) {
        const float* q = p + (k + 8 * e) * ld + n;
        split2(q[0], q[ld], f.h[e], f.m[e], f.l[e]);
    }
}
__device__ __forceinline__ void mma_bf16(float (&d)[4], const unsigned (&a)[4], const unsigned (&b)[2]) {
    asm("mma.sync.aligned.m16n8k16.row.col.f32.bf16.bf16.f32 {%0, %1, %2, %3}, {%4, %5, %6, %7}, {%8, %9}, {%0, %1, %2, %3};"
                 : "+f"(d[0]), "+f"(d[1]), "+f"(d[2]), "+f"(d[3])
                 : "r"(a[0]), "r"(a[1]), "r"(a[2]), "r"(a[3]), "r"(b[0]), "r"(b[1]));
}
// N tiles of 8 columns at once: the six additions to a tile depend on one another, those to different tiles do not
template <int N>
__device__ __forceinline__ void mma_f32(float (*d)[4], const FragA& a, const FragB* b) {
#pragma unroll
    for (int j = 0; j < N; ++j) mma_bf16(d[j], a.l, b[j].h);
#pragma unroll
    for (int j = 0; j < N; ++j) mma_bf16(d[j], a.h, b[j].l);
#pragma unroll
    for (int j = 0; j < N; ++j) mma_bf16(d[j], a.m, b[j].m);
#pragma unroll
    for (int j = 0; j < N; ++j) mma_bf16(d[j], a.m, b[j].h);
#pragma unroll
    for (int j = 0; j < N; ++j) mma_bf16(d[j], a.h, b[j].m);
#pragma unroll
    for (int j = 0; j < N; ++j) mma_bf16(d[j], a.h, b[j].h);
}
// row strides on which the fragments' accesses meet no shared-memory bank twice: pairs along a row / single numbers down a column
__host__ __device__ __forceinline__ int ld_pairs(int n) { return n + ((8 - n) & 31); }
__host__ __device__ __forceinline__ int ld_singles(int n) { return n + ((4 - n) & 15); }
__host__ __device__ __forceinline__ int up16(int n) { return (n + 15) & ~15; }

// (1) A warp's share of the lower triangle's twenty 16 x 8 tiles: up to two runs (row of tiles, first, last)
__device__ __constant__ signed char PREP_RUNS[4][2][3] = {{{3, 0, 4}, {0, 0, -1}}, {{3, 5, 7}, {0, 0, 1}}, {{2, 0, 4}, {0, 0, -1}}, {{2, 5, 5}, {1, 0, 3}}};
#define PREP_LDN 72                    // row stride of the negated A
#define PREP_LDT 24                    // of the inverted diagonal blocks
#define PREP_LDX 36                    // of a warp's 16 x 32 block of right sides
__host__ __device__ __forceinline__ int prep_second(int D, int P) {    // the q rows, later the values
    const int q = DC * ld_pairs(up16(D)), v = DC * ld_pairs(up16(P));
    return q > v ? q : v;
}
template <typename TP>
__global__ void __launch_bounds__(256, 2)
delta_prep_mma_kernel(const float* __restrict__ qkv, int C, const TP* __restrict__ proj, int ld, int a_col, int b_col,
                      const float* __restrict__ dt_bias, const float* __restrict__ A_log, float q_scale, float unit_eps,
                      const int* __restrict__ cu, int B, float* __restrict__ Wo, float* __restrict__ Uo, float* __restrict__ M,
                      float* __restrict__ rows, int H, int G, int D, int P) {
    extern __shared__ __align__(16) float sm[];
    __shared__ float s_beta[DC], s_hi[DC], s_lo[DC], s_kn[DC], s_qn[DC];
    pdl_launch_dependents();
    pdl_wait();
    int b, c;
    if (!dl_find(cu, B, blockIdx.x, &b, &c)) return;
    const int h = blockIdx.y, g = h / (H / G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gl = lane >> 2, tl = lane & 3;
    const int row0 = cu[b] + c * DC, m = min(DC, cu[b + 1] - row0);
    const int Dp = up16(D), LD = ld_pairs(Dp);
    float* K = sm;                                                // [64][LD]
    float* Q = K + DC * LD;                                       // [64][LD], then the values [64][LV]
    float* An = Q + prep_second(D, P);                            // [64][72]: -A, blocks on and below the diagonal
    float* Ti = An + DC * PREP_LDN;                               // [4][16][24]: the inverted diagonal blocks
    // a warp's eight rows are on their way together, and the numbers of the decays with them
    RawDecays raw = {};
    if (warp == 0) raw = dl_load_decays(proj, ld, a_col + h, b_col + h, row0, m, A_log + h, dt_bias + h);
    float4 q[8], k[8];
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int t = warp + 8 * i;
        q[i] = k[i] = make_float4(0.f, 0.f, 0.f, 0.f);
        if (t < m && 4 * lane < D) {
            const float* row = qkv + (size_t)(row0 + t) * C;
            q[i] = ld4(row + (size_t)g * D + 4 * lane);
            k[i] = ld4(row + (size_t)(G + g) * D + 4 * lane);
        }
    }
    if (warp == 0) dl_decays(raw, m, s_beta, s_hi, s_lo);
#pragma unroll
    for (int i = 0; i < 8; ++i) {
        const int t = warp + 8 * i;
        const float qn = q_scale / sqrtf(warp_sum(dot4(q[i], q[i])) + unit_eps), kn = 1.f / sqrtf(warp_sum(dot4(k[i], k[i])) + unit_eps);
        if (4 * lane < Dp) {                                      // (columns D .. Dp are zeros)
            st4(Q + t * LD + 4 * lane, make_float4(q[i].x * qn, q[i].y * qn, q[i].z * qn, q[i].w * qn));
            st4(K + t * LD + 4 * lane, make_float4(k[i].x * kn, k[i].y * kn, k[i].z * kn, k[i].w * kn));
        }
        if (lane == 0) { s_kn[t] = kn; s_qn[t] = qn; }
    }
    __syncthreads();
    const size_t ch = (size_t)blockIdx.x * H + h;
    if (tid < DC) dl_row_factors(rows + ch * DL_ROWS * DC, tid, m, s_qn, s_kn, s_hi, s_lo);
    {
        const int which = warp >> 2;                              // 0: k.k, 1: q.k
        const float* A = which ? Q : K;
        float* Mo = M + ch * DC * DC;
#pragma unroll 1
        for (int run = 0; run < 2; ++run) {
            const int mt = PREP_RUNS[warp & 3][run][0], n0 = PREP_RUNS[warp & 3][run][1], n1 = PREP_RUNS[warp & 3][run][2];
            if (n1 < n0) continue;
            float acc[5][4];
#pragma unroll
            for (int j = 0; j < 5; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll 1
            for (int k = 0; k < Dp; k += 16) {
                FragA a;
                frag_a_rows(a, A, LD, 16 * mt + gl, k + 2 * tl);
                if (n1 - n0 > 1) {
                    FragB f[5];
#pragma unroll
                    for (int j = 0; j < 5; ++j) frag_b_nk(f[j], K, LD, 8 * min(n0 + j, 7) + gl, k + 2 * tl);       // (behind the run: not used)
                    mma_f32<5>(acc, a, f);
                } else {
                    FragB f[2];
#pragma unroll
                    for (int j = 0; j < 2; ++j) frag_b_nk(f[j], K, LD, 8 * (n0 + j) + gl, k + 2 * tl);
                    mma_f32<2>(acc, a, f);
                }
            }
#pragma unroll
            for (int j = 0; j < 5; ++j)
                if (n0 + j <= n1) {
#pragma unroll
                    for (int half = 0; half < 2; ++half) {
                        const int t = 16 * mt + gl + 8 * half, s = 8 * (n0 + j) + 2 * tl;
                        float v[2];
#pragma unroll
                        for (int e = 0; e < 2; ++e) {
                            const float f = s + e <= t ? expf((s_hi[t] - s_hi[s + e]) + (s_lo[t] - s_lo[s + e])) : 0.f;
                            v[e] = f * acc[j][2 * half + e];
                            if (!which) v[e] = s + e < t ? -s_beta[t] * v[e] : 0.f;
                        }
                        float* dst = which ? Mo + t * DC + s : An + t * PREP_LDN + s;
                        *reinterpret_cast<float2*>(dst) = make_float2(v[0], v[1]);
                    }
                }
        }
    }
    __syncthreads();
    // the q rows are done with: their place takes the values, row by row
    const int LV = ld_pairs(up16(P));
    for (int t = warp; t < DC; t += 8)
        if (4 * lane < P) dl_copy16(Q + t * LV + 4 * lane, t < m ? qkv + (size_t)(row0 + t) * C + (size_t)2 * G * D + (size_t)h * P + 4 * lane : qkv, t < m);
    dl_commit();
    if (tid < DC) {                                               // (1 + A_ii)^-1, a thread per column
        const int i = tid >> 4, cc = tid & 15;
        float x[16];
#pragma unroll
        for (int t = 0; t < 16; ++t) {
            float v = t == cc ? 1.f : 0.f;
#pragma unroll
            for (int s = 0; s < t; ++s) v += An[(16 * i + t) * PREP_LDN + 16 * i + s] * x[s];
            x[t] = v;
            Ti[(16 * i + t) * PREP_LDT + cc] = v;
        }
    }
    dl_wait<0>();
    __syncthreads();
    // right sides in groups of 32 columns, a warp each: block row i solved by the inverse of its diagonal block, then taken off
    // the block rows below
    float* X = Ti + 4 * 16 * PREP_LDT + warp * 16 * PREP_LDX;
    const int vg = (P + 31) / 32, groups = vg + (D + 31) / 32;
#pragma unroll 1
    for (int grp = warp; grp < groups; grp += 8) {
        const bool values = grp < vg;
        const int c0 = 32 * (values ? grp : grp - vg), width = values ? P : D;
        float x[4][4][4];                                         // [block row][tile of 8 columns][fragment]
#pragma unroll
        for (int i = 0; i < 4; ++i)
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                const int t = 16 * i + gl + 8 * half;
                const float be = s_beta[t], f = values ? be : be * expf(s_hi[t] + s_lo[t]);
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    const int col = c0 + 8 * j + 2 * tl;
                    float2 v = make_float2(0.f, 0.f);
                    if (col < width) v = *reinterpret_cast<const float2*>(values ? Q + t * LV + col : K + t * LD + col);
                    x[i][j][2 * half] = f * v.x;
                    x[i][j][2 * half + 1] = f * v.y;
                }
            }
        float* dst = values ? Uo + ch * DC * P : Wo + ch * DC * D;
#pragma unroll
        for (int i = 0; i < 4; ++i) {
            FragB f[4];
            auto turn = [&]() {                                   // this block row as the second operand
                __syncwarp();
#pragma unroll
                for (int j = 0; j < 4; ++j) {
                    *reinterpret_cast<float2*>(X + gl * PREP_LDX + 8 * j + 2 * tl) = make_float2(x[i][j][0], x[i][j][1]);
                    *reinterpret_cast<float2*>(X + (gl + 8) * PREP_LDX + 8 * j + 2 * tl) = make_float2(x[i][j][2], x[i][j][3]);
                }
                __syncwarp();
#pragma unroll
                for (int j = 0; j < 4; ++j) frag_b_kn(f[j], X, PREP_LDX, 8 * j + gl, 2 * tl);
            };
            turn();
            FragA a;
            frag_a_rows(a, Ti + 16 * i * PREP_LDT, PREP_LDT, gl, 2 * tl);
#pragma unroll
            for (int j = 0; j < 4; ++j) x[i][j][0] = x[i][j][1] = x[i][j][2] = x[i][j][3] = 0.f;
            mma_f32<4>(x[i], a, f);
#pragma unroll
            for (int j = 0; j < 4; ++j) {
                const int col = c0 + 8 * j + 2 * tl;
                if (col < width) {
                    *reinterpret_cast<float2*>(dst + (size_t)(16 * i + gl) * width + col) = make_float2(x[i][j][0], x[i][j][1]);
                    *reinterpret_cast<float2*>(dst + (size_t)(16 * i + gl + 8) * width + col) = make_float2(x[i][j][2], x[i][j][3]);
                }
            }
            if (i < 3) {
                turn();
#pragma unroll
                for (int j2 = i + 1; j2 < 4; ++j2) {
                    frag_a_rows(a, An + 16 * j2 * PREP_LDN + 16 * i, PREP_LDN, gl, 2 * tl);
                    mma_f32<4>(x[j2], a, f);
                }
            }
        }
    }
}

// (2) CT value columns of one head and request: the state's tile as accumulators of the second product and, for the first, in
// shared memory.
template <int CT>
__global__ void __launch_bounds__(512)
delta_walk_mma_kernel(const float* __restrict__ qkv, int C, const float* __restrict__ W, const float* __restrict__ U0,
                      const float* __restrict__ rows, float* __restrict__ U, float* __restrict__ S0, float* __restrict__ state,
                      long long state_stride, const int* __restrict__ cu, const int* __restrict__ slots, int H, int G, int D, int P) {
    constexpr int NT = CT / 8, LDS = CT + 4, LDR = CT + 8, NH = NT / 2;
    extern __shared__ __align__(16) float sm[];
    pdl_launch_dependents();
    pdl_wait();
    const int h = blockIdx.x, b = blockIdx.y, p0 = blockIdx.z * CT;
    const int s0 = cu[b], n = cu[b + 1] - s0;
    if (n < DELTA_MIN_CHUNK) return;
    const int first = dl_first_chunk(cu, b), chunks = (n + DC - 1) / DC;
    const int g = h / (H / G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gl = lane >> 2, tl = lane & 3;
    const int Dp = up16(D), LDW = ld_pairs(Dp), LDK = ld_singles(Dp);
    const int stage = DC * LDW + DC * LDK + DC * CT + 2 * DC;
    float* Ss = sm + 2 * stage;                                   // [Dp][LDS]
    float* red = Ss + Dp * LDS;                                   // [4][64][LDR]
    float* Us = red + 4 * DC * LDR;                               // [64][LDS]: U times the k rows' factors
    if (Dp > D)                                                   // columns D .. Dp of both stages, once: no copy writes them
        for (int i = tid; i < 2 * DC * (Dp - D); i += 512) {
            const int t = i / (Dp - D), col = D + i - t * (Dp - D);
            float* w = sm + (t >= DC ? stage : 0);
            w[(t & (DC - 1)) * LDW + col] = 0.f;
            w[DC * LDW + (t & (DC - 1)) * LDK + col] = 0.f;
        }
    auto fetch = [&](int c, int buf) {
        float* w = sm + buf * stage;
        float* k = w + DC * LDW;
        float* u = k + DC * LDK;
        float* f = u + DC * CT;
        const size_t ch = (size_t)(first + c) * H + h;
        const int m = min(DC, n - c * DC);
        if (4 * lane < D) {
            const float* wg = W + ch * DC * D + 4 * lane;
            const float* kg = qkv + (size_t)(s0 + c * DC) * C + (size_t)(G + g) * D + 4 * lane;
#pragma unroll
            for (int i = 0; i < DC / 16; ++i) {
                const int t = warp + 16 * i;
                dl_copy16(w + t * LDW + 4 * lane, wg + t * D, true);
                dl_copy16(k + t * LDK + 4 * lane, t < m ? kg + (size_t)t * C : kg, t < m);
            }
        }
        if (tid < DC * CT / 4) {
            const int t = tid / (CT / 4), col = 4 * (tid % (CT / 4));
            const bool ok = p0 + col < P;
            dl_copy16(u + t * CT + col, ok ? U0 + (ch * DC + t) * P + p0 + col : U0, ok);
        }
        if (tid < 2 * DC / 4) dl_copy16(f + 4 * tid, rows + ch * DL_ROWS * DC + DC + 4 * tid, true);
    };
    // second product: rows 16 mt2 .. of the state, half of its columns' tiles from nlo on
    const int mt2 = warp & 7, nlo = (warp >> 3) * NH;
    const bool owner = 16 * mt2 < Dp;
    float* gs = state + (long long)slots[b] * state_stride + (size_t)h * D * P + p0;
    const int da = 16 * mt2 + gl, db = da + 8;
    float sr[NH][4];
#pragma unroll
    for (int j = 0; j < NH; ++j) {
        const int col = 8 * (nlo + j) + 2 * tl;
        float2 x = make_float2(0.f, 0.f), y = x;
        if (owner) {
            if (p0 + col < P) {
                if (da < D) x = *reinterpret_cast<const float2*>(gs + (size_t)da * P + col);
                if (db < D) y = *reinterpret_cast<const float2*>(gs + (size_t)db * P + col);
            }
            *reinterpret_cast<float2*>(Ss + da * LDS + col) = x;
            *reinterpret_cast<float2*>(Ss + db * LDS + col) = y;
        }
        sr[j][0] = x.x; sr[j][1] = x.y; sr[j][2] = y.x; sr[j][3] = y.y;
    }
    // first product: tokens 16 mt1 .., every fourth step of 16 rows of the state
    const int mt1 = warp & 3, kh = warp >> 2;
    fetch(0, 0);
    dl_commit();
#pragma unroll 1
    for (int c = 0; c < chunks; ++c) {
        dl_wait<0>();
        __syncthreads();
        const float* w = sm + (c & 1) * stage;
        const float* k = w + DC * LDW;
        const float* u = k + DC * LDK;
        const float* f = u + DC * CT;
        if (owner) {
            float* so = S0 + (((size_t)(first + c) * H + h) * D) * P + p0;
#pragma unroll
            for (int j = 0; j < NH; ++j) {
                const int col = 8 * (nlo + j) + 2 * tl;
                if (p0 + col < P) {
                    if (da < D) *reinterpret_cast<float2*>(so + (size_t)da * P + col) = make_float2(sr[j][0], sr[j][1]);
                    if (db < D) *reinterpret_cast<float2*>(so + (size_t)db * P + col) = make_float2(sr[j][2], sr[j][3]);
                }
            }
        }
        float acc[NT][4];
#pragma unroll
        for (int j = 0; j < NT; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
#pragma unroll 2
        for (int d = 16 * kh; d < Dp; d += 64) {
            FragA a;
            frag_a_rows(a, w, LDW, 16 * mt1 + gl, d + 2 * tl);
            FragB q[NT];
#pragma unroll
            for (int j = 0; j < NT; ++j) frag_b_kn(q[j], Ss, LDS, 8 * j + gl, d + 2 * tl);
            mma_f32<NT>(acc, a, q);
        }
#pragma unroll
        for (int j = 0; j < NT; ++j)
#pragma unroll
            for (int half = 0; half < 2; ++half)
                *reinterpret_cast<float2*>(red + (kh * DC + 16 * mt1 + gl + 8 * half) * LDR + 8 * j + 2 * tl) = make_float2(acc[j][2 * half], acc[j][2 * half + 1]);
        if (c + 1 < chunks) { fetch(c + 1, (c + 1) & 1); dl_commit(); }       // (that stage was last read before this chunk began)
        __syncthreads();
        const int m = min(DC, n - c * DC);
#pragma unroll
        for (int i = 0; i < DC * CT / 2 / 512; ++i) {             // two columns of a token a thread: the four parts, in order
            const int t = (tid + 512 * i) / (CT / 2), col = 2 * ((tid + 512 * i) % (CT / 2));
            float2 r = *reinterpret_cast<const float2*>(red + t * LDR + col);
#pragma unroll
            for (int e = 1; e < 4; ++e) {
                const float2 q = *reinterpret_cast<const float2*>(red + (e * DC + t) * LDR + col);
                r.x += q.x; r.y += q.y;
            }
            const float2 v0 = *reinterpret_cast<const float2*>(u + t * CT + col), v = make_float2(v0.x - r.x, v0.y - r.y);
            *reinterpret_cast<float2*>(Us + t * LDS + col) = make_float2(v.x * f[t], v.y * f[t]);
            if (t < m && p0 + col < P) *reinterpret_cast<float2*>(U + (size_t)(s0 + c * DC + t) * H * P + (size_t)h * P + p0 + col) = v;
        }
        __syncthreads();
        if (owner) {
            const float keep = f[DC];
#pragma unroll
            for (int j = 0; j < NH; ++j) { sr[j][0] *= keep; sr[j][1] *= keep; sr[j][2] *= keep; sr[j][3] *= keep; }
#pragma unroll
            for (int t = 0; t < DC; t += 16) {
                FragA a;
                frag_a_cols(a, k, LDK, 16 * mt2 + gl, t + 2 * tl);
                FragB q[NH];
#pragma unroll
                for (int j = 0; j < NH; ++j) frag_b_kn(q[j], Us, LDS, 8 * (nlo + j) + gl, t + 2 * tl);
                mma_f32<NH>(sr, a, q);
            }
#pragma unroll
            for (int j = 0; j < NH; ++j) {
                const int col = 8 * (nlo + j) + 2 * tl;
                *reinterpret_cast<float2*>(Ss + da * LDS + col) = make_float2(sr[j][0], sr[j][1]);
                *reinterpret_cast<float2*>(Ss + db * LDS + col) = make_float2(sr[j][2], sr[j][3]);
            }
        }
    }
    if (owner) {
#pragma unroll
        for (int j = 0; j < NH; ++j) {
            const int col = 8 * (nlo + j) + 2 * tl;
            if (p0 + col < P) {
                if (da < D) *reinterpret_cast<float2*>(gs + (size_t)da * P + col) = make_float2(sr[j][0], sr[j][1]);
                if (db < D) *reinterpret_cast<float2*>(gs + (size_t)db * P + col) = make_float2(sr[j][2], sr[j][3]);
            }
        }
    }
}

// (3) Two warps side by side on 16 tokens, NTW tiles of 8 columns each.
template <typename TP, int NTW>
__global__ void __launch_bounds__(256, 2)
delta_out_mma_kernel(const float* __restrict__ qkv, int C, const TP* __restrict__ proj, int ld, int gate_col, const float* __restrict__ M,
                     const float* __restrict__ rows, const float* __restrict__ U, const float* __restrict__ S0,
                     const float* __restrict__ norm, float eps, const int* __restrict__ cu, int B, TP* __restrict__ out, int H, int G,
                     int D, int P) {
    constexpr int COLS = 16 * NTW, LDB = COLS + 4;
    extern __shared__ __align__(16) float sm[];
    __shared__ float s_ss[2][DC];
    pdl_launch_dependents();
    pdl_wait();
    int b, c;
    if (!dl_find(cu, B, blockIdx.x, &b, &c)) return;
    const int h = blockIdx.y, g = h / (H / G), tid = threadIdx.x, warp = tid >> 5, lane = tid & 31, gl = lane >> 2, tl = lane & 3;
    const int row0 = cu[b] + c * DC, m = min(DC, cu[b + 1] - row0);
    const size_t ch = (size_t)blockIdx.x * H + h;
    const int Dp = up16(D), LD = ld_pairs(Dp), LM = DC + 8;
    float* Q = sm;                                                // [64][LD]
    float* Ms = Q + DC * LD;                                      // [64][72]
    float* Bs = Ms + DC * LM;                                     // two stages of [32][LDB]
    TP* Z = reinterpret_cast<TP*>(Bs + 2 * OUT_BK * LDB);         // the gate's numbers [64][COLS]
    const int nS = (Dp + OUT_BK - 1) / OUT_BK, tiles = nS + DC / OUT_BK;
    auto fetch = [&](int tile, int buf) {
        float* dst = Bs + buf * OUT_BK * LDB;
        const bool from_state = tile < nS;
        const int r0 = (from_state ? tile : tile - nS) * OUT_BK;
        const float* src = from_state ? S0 + ch * D * P : U + (size_t)row0 * H * P + (size_t)h * P;
        const size_t stride = from_state ? P : (size_t)H * P;
        const int last = from_state ? D : m;
#pragma unroll
        for (int i = 0; i < OUT_BK * COLS / 4 / 256; ++i) {
            const int r = (tid + 256 * i) / (COLS / 4), col = 4 * ((tid + 256 * i) % (COLS / 4));
            const bool ok = r0 + r < last && col < P;
            dl_copy16(dst + r * LDB + col, ok ? src + (size_t)(r0 + r) * stride + col : src, ok);
        }
    };
    for (int t = warp; t < DC; t += 8) {
        const bool ok = t < m && 4 * lane < D;
        if (4 * lane < Dp) dl_copy16(Q + t * LD + 4 * lane, ok ? qkv + (size_t)(row0 + t) * C + (size_t)g * D + 4 * lane : qkv, ok);
        if (lane < DC / 4) dl_copy16(Ms + t * LM + 4 * lane, M + ch * DC * DC + t * DC + 4 * lane, true);
    }
    for (int t = warp; t < DC; t += 8)
        if (4 * lane < COLS) {
            const bool ok = t < m && 4 * lane < P;
            const TP* src = ok ? proj + (size_t)(row0 + t) * ld + gate_col + (size_t)h * P + 4 * lane : proj;
            if (sizeof(TP) == 2) dl_copy8(Z + t * COLS + 4 * lane, src, ok);
            else dl_copy16(Z + t * COLS + 4 * lane, src, ok);
        }
    fetch(0, 0);
    dl_commit();
    const int mt = warp & 3, nh = warp >> 2, t0 = 16 * mt + gl;
    float acc[NTW][4];
#pragma unroll
    for (int j = 0; j < NTW; ++j) acc[j][0] = acc[j][1] = acc[j][2] = acc[j][3] = 0.f;
    const float* rw = rows + ch * DL_ROWS * DC;
#pragma unroll 1
    for (int tile = 0; tile < tiles; ++tile) {
        dl_wait<0>();
        __syncthreads();
        if (tile + 1 < tiles) { fetch(tile + 1, (tile + 1) & 1); dl_commit(); }
        if (tile == nS) {                                         // what the state gives is complete: the rows' own factors
            const float fa = rw[t0], fb = rw[t0 + 8];
#pragma unroll
            for (int j = 0; j < NTW; ++j) { acc[j][0] *= fa; acc[j][1] *= fa; acc[j][2] *= fb; acc[j][3] *= fb; }
        }
        const bool from_state = tile < nS;
        const float* A = from_state ? Q : Ms;
        const int lda = from_state ? LD : LM, k0 = (from_state ? tile : tile - nS) * OUT_BK;
        const int end = from_state ? Dp : 16 * (mt + 1);          // (of M, the blocks on and below the diagonal exist)
        const float* Bt = Bs + (tile & 1) * OUT_BK * LDB;
#pragma unroll 1
        for (int k = 0; k < OUT_BK && k0 + k < end; k += 16) {
            FragA a;
            frag_a_rows(a, A, lda, t0, k0 + k + 2 * tl);
#pragma unroll
            for (int j0 = 0; j0 < NTW; j0 += 4) {
                FragB f[4];
#pragma unroll
                for (int j = 0; j < 4; ++j) frag_b_kn(f[j], Bt, LDB, 8 * (NTW * nh + j0 + j) + gl, k + 2 * tl);
                mma_f32<4>(acc + j0, a, f);
            }
        }
    }
    float ss[2] = {0.f, 0.f};
#pragma unroll
    for (int j = 0; j < NTW; ++j)                                 // (columns behind P are zero)
#pragma unroll
        for (int half = 0; half < 2; ++half) ss[half] += acc[j][2 * half] * acc[j][2 * half] + acc[j][2 * half + 1] * acc[j][2 * half + 1];
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        ss[half] += __shfl_xor_sync(0xffffffffu, ss[half], 1);
        ss[half] += __shfl_xor_sync(0xffffffffu, ss[half], 2);
        if (tl == 0) s_ss[nh][t0 + 8 * half] = ss[half];
    }
    __syncthreads();
#pragma unroll
    for (int half = 0; half < 2; ++half) {
        const int t = t0 + 8 * half;
        if (t >= m) continue;
        const float inv = 1.f / sqrtf((s_ss[0][t] + s_ss[1][t]) / (float)P + eps);
        TP* o = out + (size_t)(row0 + t) * H * P + (size_t)h * P;
#pragma unroll
        for (int j = 0; j < NTW; ++j) {
            const int col = 8 * (NTW * nh + j) + 2 * tl;
            if (col >= P) continue;
            const float2 z = dl_load2(Z + t * COLS + col), nw = *reinterpret_cast<const float2*>(norm + col);
            dl_store2(o + col, acc[j][2 * half] * inv * nw.x * dl_silu(z.x), acc[j][2 * half + 1] * inv * nw.y * dl_silu(z.y));
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
template <int CT>
static int launch_walk_mma(const float* qkv, int C, const float* W, const float* U0, const float* rows, float* U, float* S0, float* state,
                           long long state_stride, const int* cu, const int* slots, int B, int H, int G, int D, int P, cudaStream_t s) {
    const int Dp = up16(D);
    const size_t smem = sizeof(float) * ((size_t)2 * (DC * (ld_pairs(Dp) + ld_singles(Dp)) + DC * CT + 2 * DC) + (size_t)Dp * (CT + 4)
                                         + 4 * DC * (CT + 8) + DC * (CT + 4));
    const int rc = delta_smem(delta_walk_mma_kernel<CT>, smem);
    if (rc) return rc;
    return vl_launch(delta_walk_mma_kernel<CT>, dim3(H, B, (P + CT - 1) / CT), dim3(512), smem, s, qkv, C, W, U0, rows, U, S0, state,
                     state_stride, cu, slots, H, G, D, P);
}
// MMA false: the kernels of plain float32 multiply-adds (float32 steps), else those on the tensor cores (bfloat16 steps).
template <typename TP, bool MMA>
static int launch_chunks(const float* qkv, int C, const TP* proj, int ld, int a_col, int b_col, int gate_col, const float* dt_bias,
                         const float* A_log, float q_scale, float unit_eps, const float* norm, float eps, float* state,
                         long long state_stride, const int* cu, const int* slots, int B, int chunks, float* scratch, float* U, TP* out,
                         int H, int G, int D, int P, int sms, cudaStream_t s) {
    const size_t n = (size_t)chunks * H;
    float* W = scratch;
    float* U0 = W + n * D * DC;
    float* M = U0 + n * P * DC;
    float* rows = M + n * DC * DC;
    float* S0 = rows + n * DL_ROWS * DC;
    const int Dp = up16(D);
    int rc;
    {
        auto kernel = [] { if constexpr (MMA) return delta_prep_mma_kernel<TP>; else return delta_prep_kernel<TP>; }();
        const size_t smem = sizeof(float) * (MMA ? (size_t)DC * ld_pairs(Dp) + prep_second(D, P) + DC * PREP_LDN + 4 * 16 * PREP_LDT + 8 * 16 * PREP_LDX
                                                 : (size_t)2 * DC * (D + 4) + DC * PREP_LDA);
        if ((rc = delta_smem(kernel, smem))) return rc;
        rc = vl_launch(kernel, dim3(chunks, H), dim3(256), smem, s, qkv, C, proj, ld, a_col, b_col, dt_bias, A_log, q_scale, unit_eps, cu, B,
                       W, U0, M, rows, H, G, D, P);
        if (rc) return rc;
    }
    // narrow tiles of columns while they leave an SM to every block
    const bool narrow = (long long)H * B * ((P + 15) / 16) <= sms;
#define DELTA_WALK(FN) FN(qkv, C, W, U0, rows, U, S0, state, state_stride, cu, slots, B, H, G, D, P, s)
    if constexpr (MMA) rc = narrow ? DELTA_WALK(launch_walk_mma<16>) : DELTA_WALK(launch_walk_mma<32>);
    else rc = narrow ? DELTA_WALK(launch_walk<16>) : DELTA_WALK(launch_walk<32>);
#undef DELTA_WALK
    if (rc) return rc;
    auto outputs = [&](auto kernel, size_t smem) {
        const int e = delta_smem(kernel, smem);
        if (e) return e;
        return vl_launch(kernel, dim3(chunks, H), dim3(256), smem, s, qkv, C, proj, ld, gate_col, M, rows, U, S0, norm, eps, cu, B, out, H, G, D, P);
    };
    if constexpr (MMA) {
        const size_t rest = sizeof(float) * ((size_t)DC * ld_pairs(Dp) + DC * (DC + 8));
        if (P <= 64) return outputs(delta_out_mma_kernel<TP, 4>, rest + sizeof(float) * 2 * OUT_BK * (64 + 4) + sizeof(TP) * DC * 64);
        return outputs(delta_out_mma_kernel<TP, 8>, rest + sizeof(float) * 2 * OUT_BK * (128 + 4) + sizeof(TP) * DC * 128);
    } else {
        const size_t rest = sizeof(float) * ((size_t)DC * (D + 4) + DC * (DC + 4));
        if (P <= 64) return outputs(delta_out_kernel<TP, 1>, rest + sizeof(float) * 2 * OUT_BK * 64);
        return outputs(delta_out_kernel<TP, 2>, rest + sizeof(float) * 2 * OUT_BK * 128);
    }
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
        return launch_chunks<float, false>(qkv, C, (const float*)proj, ld, a_col, b_col, gate_col, dt_bias, A_log, q_scale, unit_eps, norm, eps,
                                    state, state_stride, cu, slots, B, chunks, scratch, U, (float*)out, H, G, D, P, sms, s);
    if (dtype == VL_BF16)
        return launch_chunks<bf16, true>(qkv, C, (const bf16*)proj, ld, a_col, b_col, gate_col, dt_bias, A_log, q_scale, unit_eps, norm, eps,
                                   state, state_stride, cu, slots, B, chunks, scratch, U, (bf16*)out, H, G, D, P, sms, s);
    return VL_ERR_UNSUPPORTED;
}
