// Embedding gather and RMS norm with the residual sum folded in.
//
// The residual stream `x` is float32 in every mode.  A block hands the next
// norm a pending `delta` (the previous mixer's or feed-forward's output, in the
// activation dtype); the norm kernel adds it into `x` in float32, then norms:
//     x <- x + delta;   h = x / sqrt(mean(x^2) + eps) * w
// (formula: crates/model/src/components/norm/rms_norm.rs:26-49 of the reference).
// One block of 256 threads per row; the order of the additions of the mean is a
// function of the row length alone.
#include "common.cuh"

template <typename TW>
__global__ void embed_kernel(const int* __restrict__ ids, const TW* __restrict__ table,
                             float* __restrict__ x, int H, int V, float scale, unsigned* err) {
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x;
    const int id = ids[t];
    float* row = x + (size_t)t * H;
    if (id < 0 || id >= V) {
        if (threadIdx.x == 0) atomicOr(err, VL_DEV_BAD_TOKEN);
        for (int i = threadIdx.x; i < H; i += blockDim.x) row[i] = 0.f;
        return;
    }
    const TW* src = table + (size_t)id * H;
    for (int i = threadIdx.x; i < H; i += blockDim.x) row[i] = to_f32(src[i]) * scale;   // float32; times 1 is exact
}

// The same with a row of a second table added, hashed from the token before and this one:
//   x[t] = table[id_t] * scale + pairs[(id_(t-1) mul_prev + id_t mul_cur) mod buckets],  row `buckets` at position 0.
// The token before a portion's first one is the request's state (an int32 per slot), which the block of that token replaces
// by the portion's last token; no other block touches it.  A row at a negative position (padding of a replayed step) is
// zero and touches no state.
template <typename TW>
__global__ void embed_pair_kernel(const int* __restrict__ ids, const TW* __restrict__ table, const TW* __restrict__ pairs,
                                  float* __restrict__ x, int H, int V, float scale, int buckets, long long mul_prev,
                                  long long mul_cur, int* state, long long state_stride, const int* __restrict__ cu,
                                  const int* __restrict__ slots, const int* __restrict__ req_index,
                                  const int* __restrict__ positions, unsigned* err) {
    __shared__ int s_prev;
    pdl_launch_dependents();
    pdl_wait();
    const int t = blockIdx.x, pos = positions[t], id = ids[t];
    float* row = x + (size_t)t * H;
    if (pos < 0) {
        for (int i = threadIdx.x; i < H; i += blockDim.x) row[i] = 0.f;
        return;
    }
    if (threadIdx.x == 0) {
        const int b = req_index[t], first = cu[b];
        int prev = t > first ? ids[t - 1] : 0;
        if (t == first) {
            int* st = state + (long long)slots[b] * state_stride;
            prev = *st;
            *st = ids[cu[b + 1] - 1];
        }
        s_prev = prev;
    }
    __syncthreads();
    if (id < 0 || id >= V) {
        if (threadIdx.x == 0) atomicOr(err, VL_DEV_BAD_TOKEN);
        for (int i = threadIdx.x; i < H; i += blockDim.x) row[i] = 0.f;
        return;
    }
    const int prev = min(max(s_prev, 0), V - 1);         // (a token before that was refused was flagged at its own place)
    const long long at = pos == 0 ? buckets : (prev * mul_prev + id * mul_cur) % buckets;
    const TW* src = table + (size_t)id * H;
    const TW* add = pairs + (size_t)at * H;
    if ((H & 3) == 0) {
        for (int i = 4 * threadIdx.x; i < H; i += 4 * blockDim.x) {
            const float4 a = Quad<TW>::load(src + i), b = Quad<TW>::load(add + i);
            Quad<float>::store(row + i, make_float4(a.x * scale + b.x, a.y * scale + b.y, a.z * scale + b.z, a.w * scale + b.w));
        }
        return;
    }
    for (int i = threadIdx.x; i < H; i += blockDim.x) row[i] = to_f32(src[i]) * scale + to_f32(add[i]);
}

// rows == nullptr: row r of the output is row r of x (and x is updated in place
// when delta is given).  rows != nullptr: output row r is made from x[rows[r]]
// (+ delta[rows[r]]) and x is left untouched.
template <typename TA>
__global__ void add_rmsnorm_kernel(float* __restrict__ x, const TA* __restrict__ delta,
                                   const int* __restrict__ rows, const float* __restrict__ w,
                                   TA* __restrict__ out, int H, float eps) {
    __shared__ float scratch[32];
    const int r = blockIdx.x;
    const int src = rows ? rows[r] : r;
    float* xr = x + (size_t)src * H;
    const TA* dr = delta ? delta + (size_t)src * H : nullptr;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += 256) {
        float v = xr[i];
        if (dr) {
            v += to_f32(dr[i]);
            if (!rows) xr[i] = v;
        }
        ss += v * v;
    }
    ss = block_sum<256>(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)H + eps);
    TA* o = out + (size_t)r * H;
    for (int i = threadIdx.x; i < H; i += 256) {
        float v = xr[i];
        if (dr && rows) v += to_f32(dr[i]);
        o[i] = from_f32<TA>(v * inv * w[i]);
    }
}

// The same function with a row kept in registers: 16-byte loads, one pass over memory.
// Thread i holds the float4 pieces i, i + 256, ... of the row (H a multiple of 4, at most
// 256 * 4 * VPT values).  The sum of squares is taken piece by piece in that fixed order.
template <typename TA, int VPT>
__global__ void __launch_bounds__(256)
add_rmsnorm_vec_kernel(float* __restrict__ x, const TA* __restrict__ delta, const int* __restrict__ rows,
                       const float* __restrict__ w, TA* __restrict__ out, int H, float eps) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    const int src = rows ? rows[r] : r;
    float* xr = x + (size_t)src * H;
    const TA* dr = delta ? delta + (size_t)src * H : nullptr;
    const int H4 = H >> 2;
    float4 v[VPT];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + 256 * i;
        if (c < H4) {
            v[i] = Quad<float>::load(xr + 4 * c);
            if (dr) {
                const float4 d = Quad<TA>::load(dr + 4 * c);
                v[i].x += d.x; v[i].y += d.y; v[i].z += d.z; v[i].w += d.w;
                if (!rows) Quad<float>::store(xr + 4 * c, v[i]);
            }
            ss += v[i].x * v[i].x; ss += v[i].y * v[i].y; ss += v[i].z * v[i].z; ss += v[i].w * v[i].w;
        }
    }
    ss = block_sum<256>(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)H + eps);
    TA* o = out + (size_t)r * H;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + 256 * i;
        if (c < H4) {
            const float4 g = Quad<float>::load(w + 4 * c);
            Quad<TA>::store(o + 4 * c, make_float4(v[i].x * inv * g.x, v[i].y * inv * g.y, v[i].z * inv * g.z, v[i].w * inv * g.w));
        }
    }
}

template <typename TA>
static bool launch_rmsnorm_vec(float* x, const TA* delta, const int* rows, const float* w, TA* out, int R, int H,
                               float eps, cudaStream_t s) {
    if (H % 4) return false;
    const int pieces = (H / 4 + 255) / 256;
    if (pieces <= 1) vl_launch(add_rmsnorm_vec_kernel<TA, 1>, dim3(R), dim3(256), 0, s, x, delta, rows, w, out, H, eps);
    else if (pieces <= 2) vl_launch(add_rmsnorm_vec_kernel<TA, 2>, dim3(R), dim3(256), 0, s, x, delta, rows, w, out, H, eps);
    else if (pieces <= 4) vl_launch(add_rmsnorm_vec_kernel<TA, 4>, dim3(R), dim3(256), 0, s, x, delta, rows, w, out, H, eps);
    else if (pieces <= 8) vl_launch(add_rmsnorm_vec_kernel<TA, 8>, dim3(R), dim3(256), 0, s, x, delta, rows, w, out, H, eps);
    else return false;
    return true;
}

// y[r, c] += bias[c] for a linear layer with a bias vector: the product's result is widened, the float32
// bias added and the sum rounded once.
template <typename TA>
__global__ void add_bias_kernel(TA* __restrict__ y, const float* __restrict__ bias, size_t n, int cols) {
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) y[i] = from_f32<TA>(to_f32(y[i]) + bias[i % (size_t)cols]);
}

template <typename TI, typename TO>
__global__ void cast_kernel(const TI* __restrict__ in, TO* __restrict__ out, size_t n) {
    size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    if (i < n) out[i] = from_f32<TO>(to_f32(in[i]));
}

// Layer norm with a weight and no bias, h = (y - mean y) / sqrt(var y + eps) * w with the variance as the mean of the
// squared deviations (two passes over the row, float32), in the two places a block that norms its sub-layers'
// OUTPUTS needs it:
//   layernorm_add_kernel   x[r] += LN(y[r]) * w  (y: a sub-layer's output in the activation dtype; x: the float32
//                          stream) and, when asked, cast[r] = x[r] in the activation dtype: the next sub-layer's input
//   layernorm_rows_kernel  out[r] = LN(x[rows[r]]) * w  (the model's last norm on the rows whose logits are wanted)
// One block of 256 threads per row; the order of the sums depends on the row length alone.
template <typename TA>
__global__ void __launch_bounds__(256)
layernorm_add_kernel(const TA* __restrict__ y, const float* __restrict__ w, float eps, float* __restrict__ x,
                     TA* __restrict__ cast, int H) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    const TA* yr = y + (size_t)r * H;
    float s = 0.f;
    for (int i = threadIdx.x; i < H; i += 256) s += to_f32(yr[i]);
    const float mean = block_sum<256>(s, scratch) / (float)H;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += 256) { const float d = to_f32(yr[i]) - mean; ss += d * d; }
    const float inv = 1.0f / sqrtf(block_sum<256>(ss, scratch) / (float)H + eps);
    float* xr = x + (size_t)r * H;
    for (int i = threadIdx.x; i < H; i += 256) {
        const float v = xr[i] + (to_f32(yr[i]) - mean) * inv * w[i];
        xr[i] = v;
        if (cast) cast[(size_t)r * H + i] = from_f32<TA>(v);
    }
}

// The same with the row of y kept in registers (H a multiple of 4, at most 256 * 4 * VPT values): one read of y,
// one read and one write of x, one write of the cast, 16-byte accesses.  Thread i holds the pieces i, i + 256, ...
template <typename TA, int VPT>
__global__ void __launch_bounds__(256)
layernorm_add_vec_kernel(const TA* __restrict__ y, const float* __restrict__ w, float eps, float* __restrict__ x,
                         TA* __restrict__ cast, int H) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x, H4 = H >> 2;
    const TA* yr = y + (size_t)r * H;
    float4 v[VPT];
    float s = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + 256 * i;
        if (c < H4) {
            v[i] = Quad<TA>::load(yr + 4 * c);
            s += v[i].x; s += v[i].y; s += v[i].z; s += v[i].w;
        }
    }
    const float mean = block_sum<256>(s, scratch) / (float)H;
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + 256 * i;
        if (c < H4) {
            v[i].x -= mean; v[i].y -= mean; v[i].z -= mean; v[i].w -= mean;
            ss += v[i].x * v[i].x; ss += v[i].y * v[i].y; ss += v[i].z * v[i].z; ss += v[i].w * v[i].w;
        }
    }
    const float inv = 1.0f / sqrtf(block_sum<256>(ss, scratch) / (float)H + eps);
    float* xr = x + (size_t)r * H;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + 256 * i;
        if (c < H4) {
            const float4 g = Quad<float>::load(w + 4 * c);
            float4 o = Quad<float>::load(xr + 4 * c);
            o.x += v[i].x * inv * g.x; o.y += v[i].y * inv * g.y; o.z += v[i].z * inv * g.z; o.w += v[i].w * inv * g.w;
            Quad<float>::store(xr + 4 * c, o);
            if (cast) Quad<TA>::store(cast + (size_t)r * H + 4 * c, o);
        }
    }
}

template <typename TA>
static bool launch_layernorm_add_vec(const TA* y, const float* w, float eps, float* x, TA* cast, int R, int H, cudaStream_t s) {
    if (H % 4) return false;
    const int pieces = (H / 4 + 255) / 256;
    if (pieces <= 1) vl_launch(layernorm_add_vec_kernel<TA, 1>, dim3(R), dim3(256), 0, s, y, w, eps, x, cast, H);
    else if (pieces <= 2) vl_launch(layernorm_add_vec_kernel<TA, 2>, dim3(R), dim3(256), 0, s, y, w, eps, x, cast, H);
    else if (pieces <= 4) vl_launch(layernorm_add_vec_kernel<TA, 4>, dim3(R), dim3(256), 0, s, y, w, eps, x, cast, H);
    else if (pieces <= 8) vl_launch(layernorm_add_vec_kernel<TA, 8>, dim3(R), dim3(256), 0, s, y, w, eps, x, cast, H);
    else return false;
    return true;
}

template <typename TA>
__global__ void __launch_bounds__(256)
layernorm_rows_kernel(const float* __restrict__ x, const int* __restrict__ rows, const float* __restrict__ w,
                      float eps, TA* __restrict__ out, int H) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    const float* xr = x + (size_t)(rows ? rows[r] : r) * H;
    float s = 0.f;
    for (int i = threadIdx.x; i < H; i += 256) s += xr[i];
    const float mean = block_sum<256>(s, scratch) / (float)H;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += 256) { const float d = xr[i] - mean; ss += d * d; }
    const float inv = 1.0f / sqrtf(block_sum<256>(ss, scratch) / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += 256) out[(size_t)r * H + i] = from_f32<TA>((xr[i] - mean) * inv * w[i]);
}

extern "C" int vl_layernorm_add(const void* y, int act_dtype, const float* w, float eps, float* x, void* cast,
                                int R, int H, void* stream) {
    if (R <= 0) return VL_OK;
    if (H <= 0) return VL_ERR_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    if (act_dtype == VL_F32) {
        if (launch_layernorm_add_vec<float>((const float*)y, w, eps, x, (float*)cast, R, H, s)) return vl_launch_status();
        return vl_launch(layernorm_add_kernel<float>, dim3(R), dim3(256), 0, s, (const float*)y, w, eps, x, (float*)cast, H);
    }
    if (act_dtype == VL_BF16) {
        if (launch_layernorm_add_vec<bf16>((const bf16*)y, w, eps, x, (bf16*)cast, R, H, s)) return vl_launch_status();
        return vl_launch(layernorm_add_kernel<bf16>, dim3(R), dim3(256), 0, s, (const bf16*)y, w, eps, x, (bf16*)cast, H);
    }
    return VL_ERR_UNSUPPORTED;
}

extern "C" int vl_layernorm_rows(const float* x, const int* rows, const float* w, float eps, void* out, int act_dtype,
                                 int R, int H, void* stream) {
    if (R <= 0) return VL_OK;
    if (H <= 0) return VL_ERR_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    if (act_dtype == VL_F32)
        return vl_launch(layernorm_rows_kernel<float>, dim3(R), dim3(256), 0, s, x, rows, w, eps, (float*)out, H);
    if (act_dtype == VL_BF16)
        return vl_launch(layernorm_rows_kernel<bf16>, dim3(R), dim3(256), 0, s, x, rows, w, eps, (bf16*)out, H);
    return VL_ERR_UNSUPPORTED;
}

// RMS norm of a sub-layer's OUTPUT added into the stream with a factor: x[r] += mult * (y[r] / sqrt(mean(y[r]^2) + eps) * w)
// (y in the activation dtype, x the float32 stream, everything between in float32) and, when asked, cast[r] = x[r] in
// the activation dtype: the next sub-layer's input.  `bias` (or null): a vector added to every row of y first, in float32
// (the bias of the product that made y, left to this kernel).  The row of y is kept in registers where it fits (H a multiple of
// 4, at most 256 * 4 * VPT values), else read twice.  The order of the sums depends on the row length alone.
// With a second row y2 the normed row is s1 * y + s2 * y2, or, given weights w1 and w2, s1 * n(y) w1 + s2 * n(y2) w2 with
// n(y) = y / sqrt(mean(y^2) + eps): two sub-layers side by side, each normed by itself before they are added.
template <typename TA>
__global__ void __launch_bounds__(256)
rmsnorm_add_kernel(const TA* __restrict__ y, const float* __restrict__ bias, const float* __restrict__ w, float eps, float mult,
                   float* __restrict__ x, TA* __restrict__ cast, int H, const TA* __restrict__ y2, float s1, float s2,
                   const float* __restrict__ w1, const float* __restrict__ w2) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    const TA* yr = y + (size_t)r * H;
    const TA* y2r = y2 ? y2 + (size_t)r * H : nullptr;          // the normed row is s1 * y + s2 * y2 (two sub-layers side by side)
    float f1 = s1, f2 = s2;
    if (w1) {                                                    // ... each normed by itself first
        float sa = 0.f, sb = 0.f;
        for (int i = threadIdx.x; i < H; i += 256) { const float u = to_f32(yr[i]), v = to_f32(y2r[i]); sa += u * u; sb += v * v; }
        f1 = s1 / sqrtf(block_sum<256>(sa, scratch) / (float)H + eps);
        f2 = s2 / sqrtf(block_sum<256>(sb, scratch) / (float)H + eps);
    }
    auto row = [&](int i) {
        float d = to_f32(yr[i]);
        if (y2r) d = w1 ? f1 * d * w1[i] + f2 * to_f32(y2r[i]) * w2[i] : s1 * d + s2 * to_f32(y2r[i]);
        return d + (bias ? bias[i] : 0.f);
    };
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += 256) {
        const float d = row(i);
        ss += d * d;
    }
    const float inv = 1.0f / sqrtf(block_sum<256>(ss, scratch) / (float)H + eps);
    float* xr = x + (size_t)r * H;
    for (int i = threadIdx.x; i < H; i += 256) {
        const float d = row(i);
        const float v = xr[i] + mult * (d * inv * w[i]);
        xr[i] = v;
        if (cast) cast[(size_t)r * H + i] = from_f32<TA>(v);
    }
}

template <typename TA, int VPT, bool NORMED>
__global__ void __launch_bounds__(256)
rmsnorm_add_vec_kernel(const TA* __restrict__ y, const float* __restrict__ bias, const float* __restrict__ w, float eps, float mult,
                       float* __restrict__ x, TA* __restrict__ cast, int H, const TA* __restrict__ y2, float s1, float s2,
                   const float* __restrict__ w1, const float* __restrict__ w2) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x, H4 = H >> 2;
    const TA* yr = y + (size_t)r * H;
    const TA* y2r = y2 ? y2 + (size_t)r * H : nullptr;          // the normed row is s1 * y + s2 * y2
    float4 v[VPT];
    float ss = 0.f;
    if constexpr (NORMED) {                                      // both normed by themselves first (a kernel of its own: it holds two rows)
        float4 u[VPT];
        float sa = 0.f, sb = 0.f;
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
            const int c = threadIdx.x + 256 * i;
            if (c < H4) {
                v[i] = Quad<TA>::load(yr + 4 * c);
                u[i] = Quad<TA>::load(y2r + 4 * c);
                sa += v[i].x * v[i].x; sa += v[i].y * v[i].y; sa += v[i].z * v[i].z; sa += v[i].w * v[i].w;
                sb += u[i].x * u[i].x; sb += u[i].y * u[i].y; sb += u[i].z * u[i].z; sb += u[i].w * u[i].w;
            }
        }
        const float f1 = s1 / sqrtf(block_sum<256>(sa, scratch) / (float)H + eps);
        const float f2 = s2 / sqrtf(block_sum<256>(sb, scratch) / (float)H + eps);
#pragma unroll
        for (int i = 0; i < VPT; ++i) {
            const int c = threadIdx.x + 256 * i;
            if (c < H4) {
                const float4 g1 = Quad<float>::load(w1 + 4 * c), g2 = Quad<float>::load(w2 + 4 * c);
                v[i].x = f1 * v[i].x * g1.x + f2 * u[i].x * g2.x; v[i].y = f1 * v[i].y * g1.y + f2 * u[i].y * g2.y;
                v[i].z = f1 * v[i].z * g1.z + f2 * u[i].z * g2.z; v[i].w = f1 * v[i].w * g1.w + f2 * u[i].w * g2.w;
                if (bias) {
                    const float4 b = Quad<float>::load(bias + 4 * c);
                    v[i].x += b.x; v[i].y += b.y; v[i].z += b.z; v[i].w += b.w;
                }
                ss += v[i].x * v[i].x; ss += v[i].y * v[i].y; ss += v[i].z * v[i].z; ss += v[i].w * v[i].w;
            }
        }
    } else {
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + 256 * i;
        if (c < H4) {
            v[i] = Quad<TA>::load(yr + 4 * c);
            if (y2r) {
                const float4 u = Quad<TA>::load(y2r + 4 * c);
                v[i].x = s1 * v[i].x + s2 * u.x; v[i].y = s1 * v[i].y + s2 * u.y;
                v[i].z = s1 * v[i].z + s2 * u.z; v[i].w = s1 * v[i].w + s2 * u.w;
            }
            if (bias) {
                const float4 b = Quad<float>::load(bias + 4 * c);
                v[i].x += b.x; v[i].y += b.y; v[i].z += b.z; v[i].w += b.w;
            }
            ss += v[i].x * v[i].x; ss += v[i].y * v[i].y; ss += v[i].z * v[i].z; ss += v[i].w * v[i].w;
        }
    }
    }
    const float inv = 1.0f / sqrtf(block_sum<256>(ss, scratch) / (float)H + eps);
    float* xr = x + (size_t)r * H;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + 256 * i;
        if (c < H4) {
            const float4 g = Quad<float>::load(w + 4 * c);
            float4 o = Quad<float>::load(xr + 4 * c);
            o.x += mult * (v[i].x * inv * g.x); o.y += mult * (v[i].y * inv * g.y);
            o.z += mult * (v[i].z * inv * g.z); o.w += mult * (v[i].w * inv * g.w);
            Quad<float>::store(xr + 4 * c, o);
            if (cast) Quad<TA>::store(cast + (size_t)r * H + 4 * c, o);
        }
    }
}

template <typename TA>
static int launch_rmsnorm_add(const TA* y, const float* bias, const float* w, float eps, float mult, float* x, TA* cast, int R, int H,
                              const TA* y2, float s1, float s2, const float* w1, const float* w2, cudaStream_t s) {
    const int pieces = (H / 4 + 255) / 256;
#define RMS_ADD(VPT)                                                                                                                      \
    return w1 ? vl_launch(rmsnorm_add_vec_kernel<TA, VPT, true>, dim3(R), dim3(256), 0, s, y, bias, w, eps, mult, x, cast, H, y2, s1, s2, w1, w2) \
              : vl_launch(rmsnorm_add_vec_kernel<TA, VPT, false>, dim3(R), dim3(256), 0, s, y, bias, w, eps, mult, x, cast, H, y2, s1, s2, w1, w2)
    if (H % 4 == 0 && pieces <= 1) RMS_ADD(1);
    if (H % 4 == 0 && pieces <= 2) RMS_ADD(2);
    if (H % 4 == 0 && pieces <= 4) RMS_ADD(4);
    if (H % 4 == 0 && pieces <= 8) RMS_ADD(8);
#undef RMS_ADD
    return vl_launch(rmsnorm_add_kernel<TA>, dim3(R), dim3(256), 0, s, y, bias, w, eps, mult, x, cast, H, y2, s1, s2, w1, w2);
}

extern "C" int vl_rmsnorm_add(const void* y, int act_dtype, const float* bias, const float* w, float eps, float mult, float* x, void* cast,
                              int R, int H, const void* y2, float s1, float s2, const float* w1, const float* w2, void* stream) {
    if (R <= 0) return VL_OK;
    if (H <= 0 || (w1 == nullptr) != (w2 == nullptr) || (w1 && !y2)) return VL_ERR_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    if (act_dtype == VL_F32) return launch_rmsnorm_add<float>((const float*)y, bias, w, eps, mult, x, (float*)cast, R, H, (const float*)y2, s1, s2, w1, w2, s);
    if (act_dtype == VL_BF16) return launch_rmsnorm_add<bf16>((const bf16*)y, bias, w, eps, mult, x, (bf16*)cast, R, H, (const bf16*)y2, s1, s2, w1, w2, s);
    return VL_ERR_UNSUPPORTED;
}

// The sum that a stream waits for, formed by the kernel of the norm that reads it next:
//     x[r] <- (base or x)[r] + mult * (sa * a[r] + sb * b[r]) + add[r] + vec;      h[r] = x[r] / sqrt(mean(x[r]^2) + eps) * w
// a, b: the results of two sub-layers side by side (activation dtype, either may be null), sa, sb one factor per column (float32,
// null: ones); base, add: float32 rows; vec: one float32 row for all.  out null: only the sum.  rows given: output row r is made
// from source row rows[r] and x is left as it is.  A row is kept in registers where it fits (H a multiple of 4, at most
// 256 * 4 * VPT values); the order of the sums depends on the row length alone.
template <typename TA>
struct StreamSumArgs {
    const float *base, *sa, *sb, *add, *vec;
    const TA *a, *b;
    float mult;
};
template <typename TA>
__device__ __forceinline__ float stream_value(const StreamSumArgs<TA>& p, const float* x, size_t row, int i, int H) {
    const size_t at = row * H + i;
    float v = p.base ? p.base[at] : x[at];
    if (p.a) {
        float d = to_f32(p.a[at]) * (p.sa ? p.sa[i] : 1.f);
        if (p.b) d += to_f32(p.b[at]) * (p.sb ? p.sb[i] : 1.f);
        v += p.mult * d;
    }
    if (p.add) v += p.add[at];
    if (p.vec) v += p.vec[i];
    return v;
}
template <typename TA>
__global__ void __launch_bounds__(256)
stream_norm_kernel(float* __restrict__ x, const StreamSumArgs<TA> p, const int* __restrict__ rows, const float* __restrict__ w,
                   float eps, TA* __restrict__ out, int H) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x;
    const size_t src = rows ? rows[r] : r;
    float ss = 0.f;
    for (int i = threadIdx.x; i < H; i += 256) {
        const float v = stream_value(p, x, src, i, H);
        ss += v * v;
    }
    ss = block_sum<256>(ss, scratch);
    const float inv = 1.0f / sqrtf(ss / (float)H + eps);
    for (int i = threadIdx.x; i < H; i += 256) {
        const float v = stream_value(p, x, src, i, H);
        if (!rows) x[src * H + i] = v;                   // this thread alone reads or writes element i
        if (out) out[(size_t)r * H + i] = from_f32<TA>(v * inv * w[i]);
    }
}
template <typename TA, int VPT>
__global__ void __launch_bounds__(256)
stream_norm_vec_kernel(float* __restrict__ x, const StreamSumArgs<TA> p, const int* __restrict__ rows, const float* __restrict__ w,
                       float eps, TA* __restrict__ out, int H) {
    __shared__ float scratch[32];
    pdl_launch_dependents();
    pdl_wait();
    const int r = blockIdx.x, H4 = H >> 2;
    const size_t at = (size_t)(rows ? rows[r] : r) * H;
    const float* from = (p.base ? p.base : x) + at;
    float4 v[VPT];
    float ss = 0.f;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + 256 * i;
        if (c < H4) {
            v[i] = Quad<float>::load(from + 4 * c);
            if (p.a) {
                float4 d = Quad<TA>::load(p.a + at + 4 * c);
                if (p.sa) {
                    const float4 s = Quad<float>::load(p.sa + 4 * c);
                    d.x *= s.x; d.y *= s.y; d.z *= s.z; d.w *= s.w;
                }
                if (p.b) {
                    const float4 e = Quad<TA>::load(p.b + at + 4 * c);
                    const float4 s = p.sb ? Quad<float>::load(p.sb + 4 * c) : make_float4(1.f, 1.f, 1.f, 1.f);
                    d.x += e.x * s.x; d.y += e.y * s.y; d.z += e.z * s.z; d.w += e.w * s.w;
                }
                v[i].x += p.mult * d.x; v[i].y += p.mult * d.y; v[i].z += p.mult * d.z; v[i].w += p.mult * d.w;
            }
            if (p.add) {
                const float4 e = Quad<float>::load(p.add + at + 4 * c);
                v[i].x += e.x; v[i].y += e.y; v[i].z += e.z; v[i].w += e.w;
            }
            if (p.vec) {
                const float4 e = Quad<float>::load(p.vec + 4 * c);
                v[i].x += e.x; v[i].y += e.y; v[i].z += e.z; v[i].w += e.w;
            }
            if (!rows) Quad<float>::store(x + at + 4 * c, v[i]);
            ss += v[i].x * v[i].x; ss += v[i].y * v[i].y; ss += v[i].z * v[i].z; ss += v[i].w * v[i].w;
        }
    }
    if (!out) return;
    const float inv = 1.0f / sqrtf(block_sum<256>(ss, scratch) / (float)H + eps);
    TA* o = out + (size_t)r * H;
#pragma unroll
    for (int i = 0; i < VPT; ++i) {
        const int c = threadIdx.x + 256 * i;
        if (c < H4) {
            const float4 g = Quad<float>::load(w + 4 * c);
            Quad<TA>::store(o + 4 * c, make_float4(v[i].x * inv * g.x, v[i].y * inv * g.y, v[i].z * inv * g.z, v[i].w * inv * g.w));
        }
    }
}
template <typename TA>
static int launch_stream_norm(float* x, const StreamSumArgs<TA>& p, const int* rows, const float* w, float eps, TA* out, int R, int H,
                              cudaStream_t s) {
    const int pieces = (H / 4 + 255) / 256;
    const bool vec = H % 4 == 0 && (((uintptr_t)x | (uintptr_t)p.base | (uintptr_t)p.sa | (uintptr_t)p.sb | (uintptr_t)p.add |
                                     (uintptr_t)p.vec | (uintptr_t)p.a | (uintptr_t)p.b | (uintptr_t)w | (uintptr_t)out) & 15) == 0;
#define STREAM_NORM(KERNEL) return vl_launch(KERNEL, dim3(R), dim3(256), 0, s, x, p, rows, w, eps, out, H)
    if (vec && pieces <= 1) STREAM_NORM((stream_norm_vec_kernel<TA, 1>));
    if (vec && pieces <= 2) STREAM_NORM((stream_norm_vec_kernel<TA, 2>));
    if (vec && pieces <= 4) STREAM_NORM((stream_norm_vec_kernel<TA, 4>));
    if (vec && pieces <= 8) STREAM_NORM((stream_norm_vec_kernel<TA, 8>));
    STREAM_NORM(stream_norm_kernel<TA>);
#undef STREAM_NORM
}

extern "C" int vl_stream_norm(float* x, const float* base, const void* a, const float* sa, const void* b, const float* sb, float mult,
                              const float* add, const float* vec, const int* rows, const float* w, float eps, void* out, int act_dtype,
                              int R, int H, void* stream) {
    if (R <= 0) return VL_OK;
    if (H <= 0 || (b && !a) || (out && !w) || (!out && rows)) return VL_ERR_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    if (act_dtype == VL_F32)
        return launch_stream_norm<float>(x, StreamSumArgs<float>{base, sa, sb, add, vec, (const float*)a, (const float*)b, mult}, rows, w, eps,
                                         (float*)out, R, H, s);
    if (act_dtype == VL_BF16)
        return launch_stream_norm<bf16>(x, StreamSumArgs<bf16>{base, sa, sb, add, vec, (const bf16*)a, (const bf16*)b, mult}, rows, w, eps,
                                        (bf16*)out, R, H, s);
    return VL_ERR_UNSUPPORTED;
}

extern "C" int vl_embed(const int* ids, const void* table, int table_dtype, float* x,
                        int T, int H, int V, float scale, unsigned* err, void* stream) {
    if (T <= 0) return VL_OK;
    cudaStream_t s = (cudaStream_t)stream;
    if (table_dtype == VL_F32)
        vl_launch(embed_kernel<float>, dim3(T), dim3(256), 0, s, ids, (const float*)table, x, H, V, scale, err);
    else if (table_dtype == VL_BF16)
        vl_launch(embed_kernel<bf16>, dim3(T), dim3(256), 0, s, ids, (const bf16*)table, x, H, V, scale, err);
    else
        return VL_ERR_UNSUPPORTED;
    return vl_launch_status();
}

extern "C" int vl_embed_pair(const int* ids, const void* table, const void* pairs, int table_dtype, float* x, int T, int H, int V,
                             float scale, int buckets, long long mul_prev, long long mul_cur, int* state, long long state_stride,
                             const int* cu, const int* slots, const int* req_index, const int* positions, unsigned* err, void* stream) {
    if (T <= 0) return VL_OK;
    if (H <= 0 || V <= 0 || buckets <= 0 || mul_prev < 0 || mul_cur < 0 || mul_prev > 0x7fffffff || mul_cur > 0x7fffffff || state_stride < 1)
        return VL_ERR_ARGUMENT;
    if ((((uintptr_t)table | (uintptr_t)pairs | (uintptr_t)x) & 15)) return VL_ERR_ARGUMENT;
    cudaStream_t s = (cudaStream_t)stream;
    if (table_dtype == VL_F32)
        return vl_launch(embed_pair_kernel<float>, dim3(T), dim3(256), 0, s, ids, (const float*)table, (const float*)pairs, x, H, V, scale,
                         buckets, mul_prev, mul_cur, state, state_stride, cu, slots, req_index, positions, err);
    if (table_dtype == VL_BF16)
        return vl_launch(embed_pair_kernel<bf16>, dim3(T), dim3(256), 0, s, ids, (const bf16*)table, (const bf16*)pairs, x, H, V, scale,
                         buckets, mul_prev, mul_cur, state, state_stride, cu, slots, req_index, positions, err);
    return VL_ERR_UNSUPPORTED;
}

extern "C" int vl_add_rmsnorm(float* x, const void* delta, const int* rows, const float* w, void* out,
                              int act_dtype, int R, int H, float eps, void* stream) {
    if (R <= 0) return VL_OK;
    cudaStream_t s = (cudaStream_t)stream;
    if (act_dtype == VL_F32) {
        if (!launch_rmsnorm_vec<float>(x, (const float*)delta, rows, w, (float*)out, R, H, eps, s))
            add_rmsnorm_kernel<float><<<R, 256, 0, s>>>(x, (const float*)delta, rows, w, (float*)out, H, eps);
    } else if (act_dtype == VL_BF16) {
        if (!launch_rmsnorm_vec<bf16>(x, (const bf16*)delta, rows, w, (bf16*)out, R, H, eps, s))
            add_rmsnorm_kernel<bf16><<<R, 256, 0, s>>>(x, (const bf16*)delta, rows, w, (bf16*)out, H, eps);
    } else {
        return VL_ERR_UNSUPPORTED;
    }
    return vl_launch_status();
}

extern "C" int vl_add_bias(void* y, int act_dtype, const float* bias, long long rows, int cols, void* stream) {
    if (rows <= 0 || cols <= 0) return VL_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const size_t n = (size_t)rows * (size_t)cols;
    const unsigned blocks = (unsigned)((n + 255) / 256);
    if (act_dtype == VL_F32)
        add_bias_kernel<float><<<blocks, 256, 0, s>>>((float*)y, bias, n, cols);
    else if (act_dtype == VL_BF16)
        add_bias_kernel<bf16><<<blocks, 256, 0, s>>>((bf16*)y, bias, n, cols);
    else
        return VL_ERR_UNSUPPORTED;
    return vl_launch_status();
}

extern "C" int vl_cast(const void* in, int in_dtype, void* out, int out_dtype, long long n, void* stream) {
    if (n <= 0) return VL_OK;
    cudaStream_t s = (cudaStream_t)stream;
    const unsigned blocks = (unsigned)((n + 255) / 256);
    if (in_dtype == VL_F32 && out_dtype == VL_BF16)
        cast_kernel<float, bf16><<<blocks, 256, 0, s>>>((const float*)in, (bf16*)out, (size_t)n);
    else if (in_dtype == VL_BF16 && out_dtype == VL_F32)
        cast_kernel<bf16, float><<<blocks, 256, 0, s>>>((const bf16*)in, (float*)out, (size_t)n);
    else
        return VL_ERR_UNSUPPORTED;
    return vl_launch_status();
}
