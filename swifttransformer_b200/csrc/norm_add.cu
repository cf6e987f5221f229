// Two elementwise kernels of blocks that normalise a sub-layer's OUTPUT before the residual sum, and of
// gated feed-forwards.
//
// norm_add:   x[r] += mult * gain * y[r] / sqrt(mean(y[r]^2) + eps)      (gain: one number, read from the device)
//             optionally act[r] = x[r] in the activation type, for the sub-layer that reads x next.
//             x is the float residual stream; statistics and the sum are float for every storage type.
// gated_norm_add: u = y[r] * sigmoid(g[r] + b)  (g: gate logits, or none);  x[r] += gain * u / sqrt(mean(u^2) + eps)
//             with a gain per column, and in the same pass what reads x next: act[r] = RMS norm of the new x with a
//             weight (next_gain), or the new x itself, in the activation type.
// side_input: out[r][j] = gelu_tanh(s[r][j]) * table[id[r]][col0 + j]    (a layer's own input looked up by token)
// slice_rows: out[r][j] = in[r][col0 + j], float columns of a wider tensor in the activation type
// gated_act:  out[r][j] = act(gu[r][j]) * gu[r][inner + j]               (gu = the fused gate | up product)
#include "common.cuh"

template <typename T, typename TO, bool VEC>
__global__ void __launch_bounds__(256)
norm_add_kernel(float* __restrict__ x, const T* __restrict__ y, const float* __restrict__ gain, float mult, float eps,
                int width, const int* __restrict__ positions, TO* __restrict__ act) {
    __shared__ float scratch[32];
    const float g = gain[0];                             // a weight: fetched before the wait
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    const int r = blockIdx.x;
    if (positions && positions[r] < 0) return;          // padding token of a fixed-shape step
    const T* yr = y + (size_t)r * width;
    float* xr = x + (size_t)r * width;
    float ss = 0.f;
    if (VEC) {
        for (int e = threadIdx.x * 4; e < width; e += blockDim.x * 4) {
            const float4 v = load4_cg(yr + e);
            ss = fmaf(v.x, v.x, fmaf(v.y, v.y, fmaf(v.z, v.z, fmaf(v.w, v.w, ss))));
        }
    } else {
        for (int e = threadIdx.x; e < width; e += blockDim.x) {
            const float v = load1_cg(yr + e);
            ss = fmaf(v, v, ss);
        }
    }
    ss = block_sum(ss, scratch);
    const float k = rsqrtf(ss / (float)width + eps) * g * mult;
    if (VEC) {
        for (int e = threadIdx.x * 4; e < width; e += blockDim.x * 4) {
            const float4 v = load4_cg(yr + e), o = load4_cg(xr + e);
            const float4 n = make_float4(o.x + k * v.x, o.y + k * v.y, o.z + k * v.z, o.w + k * v.w);
            store4(xr + e, n);
            if (act) store4(act + (size_t)r * width + e, n);
        }
    } else {
        for (int e = threadIdx.x; e < width; e += blockDim.x) {
            const float v = __ldcg(xr + e) + k * load1_cg(yr + e);
            xr[e] = v;
            if (act) act[(size_t)r * width + e] = from_f32<TO>(v);
        }
    }
}

ST_EXPORT int st_norm_add(float* x, const void* y, const float* gain, float mult, float eps, int n_rows, int width,
                          const int* positions, void* act, int dtype, void* stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0) return ST_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = width % 4 == 0 && aligned16(x) && aligned16(y) && aligned16(act);
    int block = ((vec ? width / 4 : width) + 31) / 32 * 32;
    if (block > 256) block = 256;
#define NA_LAUNCH(T, VEC)                                                                                         \
    return st_launch_pdl("norm_add", norm_add_kernel<T, T, VEC>, dim3(n_rows), dim3(block), 0, s, x, (const T*)y, gain, \
                         mult, eps, width, positions, (T*)act)
    if (dtype == 0) {
        if (vec) NA_LAUNCH(float, true);
        NA_LAUNCH(float, false);
    } else if (dtype == 1) {
        if (vec) NA_LAUNCH(bf16, true);
        NA_LAUNCH(bf16, false);
    }
#undef NA_LAUNCH
    return ST_ERR_BAD_DTYPE;
}

// VPT > 0: the row lives in registers, VPT vectors of four per thread (width % 4 == 0, 16-byte aligned rows);
// VPT == 0: any width, the row in shared memory.  A block takes one row after another.
template <typename TY, typename T, int VPT>
__global__ void __launch_bounds__(512)
gated_norm_add_kernel(float* __restrict__ x, const TY* __restrict__ y, const T* __restrict__ g, int g_ld,
                      const float* __restrict__ gb, const float* __restrict__ gain, float eps,
                      const float* __restrict__ next_gain, float next_eps, int n_rows, int width,
                      const int* __restrict__ positions, T* __restrict__ act) {
    extern __shared__ __align__(16) float gn_row[];
    __shared__ float scratch[32];
    ST_PDL_TRIGGER();
    ST_PDL_WAIT();
    for (int r = blockIdx.x; r < n_rows; r += gridDim.x) {
        if (positions && positions[r] < 0) continue;        // padding token of a fixed-shape step
        const TY* yr = y + (size_t)r * width;
        const T* gr = g ? g + (size_t)r * g_ld : nullptr;
        float* xr = x + (size_t)r * width;
        T* ar = act ? act + (size_t)r * width : nullptr;
        float ss = 0.f;
        if constexpr (VPT > 0) {
            float4 u[VPT], xo[VPT];
#pragma unroll
            for (int j = 0; j < VPT; ++j) {
                const int e = 4 * (threadIdx.x + j * blockDim.x);
                u[j] = xo[j] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (e >= width) continue;
                u[j] = load4_cg(yr + e);
                xo[j] = load4_cg(xr + e);
                if (gr) {
                    const float4 q = load4_cg(gr + e), b = load4(gb + e);
                    u[j].x *= 1.f / (1.f + expf(-(q.x + b.x)));
                    u[j].y *= 1.f / (1.f + expf(-(q.y + b.y)));
                    u[j].z *= 1.f / (1.f + expf(-(q.z + b.z)));
                    u[j].w *= 1.f / (1.f + expf(-(q.w + b.w)));
                }
                ss += (u[j].x * u[j].x + u[j].y * u[j].y) + (u[j].z * u[j].z + u[j].w * u[j].w);
            }
            const float k = 1.f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
            float s2 = 0.f;
#pragma unroll
            for (int j = 0; j < VPT; ++j) {
                const int e = 4 * (threadIdx.x + j * blockDim.x);
                if (e >= width) continue;
                const float4 w = load4(gain + e);
                xo[j] = make_float4(xo[j].x + u[j].x * k * w.x, xo[j].y + u[j].y * k * w.y, xo[j].z + u[j].z * k * w.z,
                                    xo[j].w + u[j].w * k * w.w);
                store4(xr + e, xo[j]);
                s2 += (xo[j].x * xo[j].x + xo[j].y * xo[j].y) + (xo[j].z * xo[j].z + xo[j].w * xo[j].w);
            }
            if (!ar) continue;
            const float k2 = next_gain ? 1.f / sqrtf(block_sum(s2, scratch) / (float)width + next_eps) : 1.f;
#pragma unroll
            for (int j = 0; j < VPT; ++j) {
                const int e = 4 * (threadIdx.x + j * blockDim.x);
                if (e >= width) continue;
                const float4 w = next_gain ? load4(next_gain + e) : make_float4(1.f, 1.f, 1.f, 1.f);
                store4(ar + e, make_float4(xo[j].x * k2 * w.x, xo[j].y * k2 * w.y, xo[j].z * k2 * w.z, xo[j].w * k2 * w.w));
            }
        } else {
            // (a thread reads back only what it wrote itself)
            for (int e = threadIdx.x; e < width; e += blockDim.x) {
                float v = load1_cg(yr + e);
                if (gr) v *= 1.f / (1.f + expf(-(load1_cg(gr + e) + gb[e])));
                gn_row[e] = v;
                ss = fmaf(v, v, ss);
            }
            const float k = 1.f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
            float s2 = 0.f;
            for (int e = threadIdx.x; e < width; e += blockDim.x) {
                const float v = __ldcg(xr + e) + gn_row[e] * k * gain[e];
                xr[e] = v;
                gn_row[e] = v;
                s2 = fmaf(v, v, s2);
            }
            if (!ar) continue;
            const float k2 = next_gain ? 1.f / sqrtf(block_sum(s2, scratch) / (float)width + next_eps) : 1.f;
            for (int e = threadIdx.x; e < width; e += blockDim.x)
                ar[e] = from_f32<T>(gn_row[e] * k2 * (next_gain ? next_gain[e] : 1.f));
        }
    }
}

// y: [n_rows, width] float (y_f32) or the storage type; g: gate logits at g[r * g_ld + e] in the storage type with the
// float bias gb, or null; act null: only x is updated
ST_EXPORT int st_gated_norm_add(float* x, const void* y, int y_f32, const void* g, int g_ld, const float* gb,
                                const float* gain, float eps, const float* next_gain, float next_eps, int n_rows,
                                int width, const int* positions, void* act, int dtype, void* stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0 || (g && !gb) || !gain) return ST_ERR_BAD_ARG;
    if ((size_t)width * sizeof(float) > 200 * 1024) return ST_ERR_TOO_LARGE;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = width % 4 == 0 && width <= 8192 && (!g || g_ld % 4 == 0) && aligned16(x) && aligned16(y) && aligned16(g) &&
                     aligned16(gb) && aligned16(gain) && aligned16(next_gain) && aligned16(act);
    const int vpt = !vec ? 0 : width <= 2048 ? 1 : width <= 4096 ? 2 : 4;
    int block = vpt ? (width / 4 / vpt + 31) / 32 * 32 : 256;
    if (vpt && width % (4 * vpt)) block += 32;
    if (block > 512) block = 512;
    const size_t smem = vpt ? 0 : (size_t)width * sizeof(float);
    int grid = st_sm_count() * 4;
    if (grid > n_rows) grid = n_rows;
#define GN_LAUNCH(TY, T, VPT)                                                                                             \
    do {                                                                                                                  \
        auto kern = gated_norm_add_kernel<TY, T, VPT>;                                                                    \
        if (smem > 40 * 1024) {                                                                                           \
            cudaError_t e = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);           \
            if (e != cudaSuccess) return (int)e;                                                                          \
        }                                                                                                                 \
        return st_launch_pdl("gated_norm_add", kern, dim3(grid), dim3(block), smem, s, x, (const TY*)y, (const T*)g, g_ld, gb, \
                             gain, eps, next_gain, next_eps, n_rows, width, positions, (T*)act);                          \
    } while (0)
#define GN_PICK(TY, T)                                                                     \
    do {                                                                                   \
        if (vpt == 0) GN_LAUNCH(TY, T, 0);                                                 \
        if (vpt == 1) GN_LAUNCH(TY, T, 1);                                                 \
        if (vpt == 2) GN_LAUNCH(TY, T, 2);                                                 \
        GN_LAUNCH(TY, T, 4);                                                               \
    } while (0)
    if (dtype == 0) GN_PICK(float, float);
    if (dtype != 1) return ST_ERR_BAD_DTYPE;
    if (y_f32) GN_PICK(float, bf16);
    GN_PICK(bf16, bf16);
#undef GN_PICK
#undef GN_LAUNCH
}

template <typename T>
__global__ void side_input_kernel(const float* __restrict__ s, const T* __restrict__ table, long long table_ld, int col0,
                                  const int* __restrict__ ids, T* __restrict__ out, int dim, int total) {
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < total; i += gridDim.x * blockDim.x) {
        const int r = i / dim, j = i % dim;
        const float e = to_f32(table[(long long)ids[r] * table_ld + col0 + j]);
        out[i] = from_f32<T>(apply_act(__ldcg(s + i), 3) * e);
    }
}

ST_EXPORT int st_side_input(const float* s, const void* table, long long table_ld, int col0, const int* ids, void* out,
                            int n_rows, int dim, int dtype, void* stream) {
    if (n_rows <= 0) return 0;
    if (dim <= 0 || col0 < 0 || col0 + dim > table_ld) return ST_ERR_BAD_ARG;
    const long long total = (long long)n_rows * dim;
    if (total > 0x7fffffffLL) return ST_ERR_TOO_LARGE;
    int grid = (int)((total + 255) / 256);
    if (grid > st_sm_count() * 8) grid = st_sm_count() * 8;
    cudaStream_t st = (cudaStream_t)stream;
    if (dtype == 0)
        return st_launch_pdl("side_input", side_input_kernel<float>, dim3(grid), dim3(256), 0, st, s, (const float*)table, table_ld,
                             col0, ids, (float*)out, dim, (int)total);
    if (dtype == 1)
        return st_launch_pdl("side_input", side_input_kernel<bf16>, dim3(grid), dim3(256), 0, st, s, (const bf16*)table, table_ld,
                             col0, ids, (bf16*)out, dim, (int)total);
    return ST_ERR_BAD_DTYPE;
}

template <typename T>
__global__ void slice_rows_kernel(const float* __restrict__ in, int ld, int col0, T* __restrict__ out, int cols, int total) {
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    for (int i = blockIdx.x * blockDim.x + threadIdx.x; i < total; i += gridDim.x * blockDim.x)
        out[i] = from_f32<T>(__ldcg(in + (size_t)(i / cols) * ld + col0 + i % cols));
}

ST_EXPORT int st_slice_rows(const float* in, int ld, int col0, void* out, int n_rows, int cols, int dtype, void* stream) {
    if (n_rows <= 0) return 0;
    if (cols <= 0 || col0 < 0 || col0 + cols > ld) return ST_ERR_BAD_ARG;
    const long long total = (long long)n_rows * cols;
    if (total > 0x7fffffffLL) return ST_ERR_TOO_LARGE;
    int grid = (int)((total + 255) / 256);
    if (grid > st_sm_count() * 8) grid = st_sm_count() * 8;
    cudaStream_t s = (cudaStream_t)stream;
    if (dtype == 0)
        return st_launch_pdl("slice_rows", slice_rows_kernel<float>, dim3(grid), dim3(256), 0, s, in, ld, col0, (float*)out, cols,
                             (int)total);
    if (dtype == 1)
        return st_launch_pdl("slice_rows", slice_rows_kernel<bf16>, dim3(grid), dim3(256), 0, s, in, ld, col0, (bf16*)out, cols,
                             (int)total);
    return ST_ERR_BAD_DTYPE;
}

// VEC: inner % 8 == 0 and 16-byte aligned rows: eight outputs per thread
template <typename T, bool VEC>
__global__ void gated_act_kernel(const T* __restrict__ gu, int ld, T* __restrict__ out, int inner, size_t total, int act) {
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    if (VEC) {
        for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 8; i < total; i += stride * 8) {
            const size_t r = i / inner, j = i % inner;
            const T* row = gu + r * ld + j;
            const float4 g0 = load4_cg(row), g1 = load4_cg(row + 4), u0 = load4_cg(row + inner), u1 = load4_cg(row + inner + 4);
            store4(out + i, make_float4(apply_act(g0.x, act) * u0.x, apply_act(g0.y, act) * u0.y,
                                        apply_act(g0.z, act) * u0.z, apply_act(g0.w, act) * u0.w));
            store4(out + i + 4, make_float4(apply_act(g1.x, act) * u1.x, apply_act(g1.y, act) * u1.y,
                                            apply_act(g1.z, act) * u1.z, apply_act(g1.w, act) * u1.w));
        }
    } else {
        for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += stride) {
            const size_t r = i / inner, j = i % inner;
            const T* row = gu + r * ld;
            out[i] = from_f32<T>(apply_act(load1_cg(row + j), act) * load1_cg(row + inner + j));
        }
    }
}

// gu: [n_rows, ld], gate then up in the first 2 * inner columns
ST_EXPORT int st_gated_act(const void* gu, int ld, void* out, int n_rows, int inner, int act, int dtype, void* stream) {
    if (n_rows <= 0) return 0;
    if (inner <= 0 || ld < 2 * inner || act < 0 || act > 5) return ST_ERR_BAD_ARG;
    const size_t total = (size_t)n_rows * inner;
    const bool vec = inner % 8 == 0 && ld % 8 == 0 && aligned16(gu) && aligned16(out);
    const size_t work = vec ? total / 8 : total;
    int grid = (int)((work + 255) / 256);
    if (grid > st_sm_count() * 16) grid = st_sm_count() * 16;
    cudaStream_t s = (cudaStream_t)stream;
#define GA_LAUNCH(T, VEC)                                                                                         \
    return st_launch_pdl("gated_act", gated_act_kernel<T, VEC>, dim3(grid), dim3(256), 0, s, (const T*)gu, ld, (T*)out, inner, \
                         total, act)
    if (dtype == 0) {
        if (vec) GA_LAUNCH(float, true);
        GA_LAUNCH(float, false);
    } else if (dtype == 1) {
        if (vec) GA_LAUNCH(bf16, true);
        GA_LAUNCH(bf16, false);
    }
#undef GA_LAUNCH
    return ST_ERR_BAD_DTYPE;
}

// The gated unit with limits, from the fused gate | up product gu [rows, 2 * inner] and its bias (float
// [2 * inner] or null):  g = min(gate + b_g, limit), u = clamp(up + b_u, -limit, limit),
// out = g * sigmoid(alpha * g) * (u + shift).  limit <= 0: no limits.
__device__ __forceinline__ float gated_clamped_one(float g, float u, float limit, float alpha, float shift) {
    if (limit > 0.f) { g = fminf(g, limit); u = fminf(fmaxf(u, -limit), limit); }
    return g / (1.f + expf(-alpha * g)) * (u + shift);
}

// VEC: inner % 8 == 0 and 16-byte aligned rows: eight outputs per thread
template <typename T, bool VEC>
__global__ void gated_clamped_act_kernel(const T* __restrict__ gu, const float* __restrict__ bias, T* __restrict__ out,
                                         int inner, size_t total, float limit, float alpha, float shift) {
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    const size_t stride = (size_t)gridDim.x * blockDim.x;
    if (VEC) {
        for (size_t i = ((size_t)blockIdx.x * blockDim.x + threadIdx.x) * 8; i < total; i += stride * 8) {
            const size_t r = i / inner, j = i % inner;
            const T* row = gu + r * 2 * inner + j;
#pragma unroll
            for (int half = 0; half < 2; ++half) {
                float4 g = load4_cg(row + 4 * half), u = load4_cg(row + inner + 4 * half);
                if (bias) {
                    g = add4(g, load4(bias + j + 4 * half));
                    u = add4(u, load4(bias + inner + j + 4 * half));
                }
                store4(out + i + 4 * half, make_float4(gated_clamped_one(g.x, u.x, limit, alpha, shift),
                                                       gated_clamped_one(g.y, u.y, limit, alpha, shift),
                                                       gated_clamped_one(g.z, u.z, limit, alpha, shift),
                                                       gated_clamped_one(g.w, u.w, limit, alpha, shift)));
            }
        }
    } else {
        for (size_t i = (size_t)blockIdx.x * blockDim.x + threadIdx.x; i < total; i += stride) {
            const size_t r = i / inner, j = i % inner;
            const T* row = gu + r * 2 * inner;
            float g = load1_cg(row + j), u = load1_cg(row + inner + j);
            if (bias) { g += bias[j]; u += bias[inner + j]; }
            out[i] = from_f32<T>(gated_clamped_one(g, u, limit, alpha, shift));
        }
    }
}

ST_EXPORT int st_gated_clamped_act(const void* gu, const float* bias, void* out, int n_rows, int inner, float limit,
                                   float alpha, float shift, int dtype, void* stream) {
    if (n_rows <= 0) return 0;
    if (inner <= 0) return ST_ERR_BAD_ARG;
    const size_t total = (size_t)n_rows * inner;
    const bool vec = inner % 8 == 0 && aligned16(gu) && aligned16(out) && (!bias || aligned16(bias));
    const size_t work = vec ? total / 8 : total;
    int grid = (int)((work + 255) / 256);
    if (grid > st_sm_count() * 16) grid = st_sm_count() * 16;
    cudaStream_t s = (cudaStream_t)stream;
#define GC_LAUNCH(T, VEC)                                                                                          \
    return st_launch_pdl("gated_clamped", gated_clamped_act_kernel<T, VEC>, dim3(grid), dim3(256), 0, s, (const T*)gu, \
                         bias, (T*)out, inner, total, limit, alpha, shift)
    if (dtype == 0) {
        if (vec) GC_LAUNCH(float, true);
        GC_LAUNCH(float, false);
    } else if (dtype == 1) {
        if (vec) GC_LAUNCH(bf16, true);
        GC_LAUNCH(bf16, false);
    }
#undef GC_LAUNCH
    return ST_ERR_BAD_DTYPE;
}
