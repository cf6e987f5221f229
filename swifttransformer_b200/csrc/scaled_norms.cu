// The residual sum of two sub-layers that read the same rows, with a factor per column for each, and the norms that read
// the new rows next, in one pass:
//
//   v      = x[r] + e[r] + (s1 * a[r] + s2 * f[r])          each of e, a, f may be absent
//   x[r]   <- v
//   out1[r] = v / sqrt(mean(v^2) + eps) * w1                out2 likewise with w2 (the statistics are shared)
//
// x, a, e are float rows.  f is a float row, or the weighted sum of a token's experts taken where it is needed:
// f[r] = sum_k weight[r,k] * y[place[r,k]] + (sum of the weights of the identity choices) * h[r]  (see moe.cu).
// With `rows` only the rows[r] are read, x is left alone and the results stand in the order of `rows` (the rows whose
// logits are wanted, at the end of a model).
#include "moe.cuh"

#define SN_MAX_TOP 64

struct ScaledSum {
    const float *a, *s1, *f, *s2, *e;
    const void *y, *h;                 // experts' rows in sorted order, the rows the identity choices stand for
    const int *place, *experts;
    const float* weights;
    int top, n_real;
};

// VPT > 0: the row lives in registers, VPT vectors of four per thread; VPT == 0: any width, the row in shared memory.
template <typename T, int VPT>
__global__ void __launch_bounds__(512)
scaled_sum_norms_kernel(float* __restrict__ x, ScaledSum p, const float* __restrict__ w1, const float* __restrict__ w2,
                        float eps, const int* __restrict__ rows, int n_rows, int width,
                        const int* __restrict__ positions, T* __restrict__ out1, T* __restrict__ out2) {
    extern __shared__ __align__(16) float sn_row[];
    __shared__ float scratch[32];
    __shared__ int s_place[SN_MAX_TOP];
    __shared__ float s_weight[SN_MAX_TOP];
    __shared__ float s_identity;
    ST_PDL_TRIGGER();
    ST_PDL_WAIT();
    const T* y = reinterpret_cast<const T*>(p.y);
    const T* h = reinterpret_cast<const T*>(p.h);
    const bool pending = p.a || p.f || p.e || y;
    for (int r = blockIdx.x; r < n_rows; r += gridDim.x) {
        const int i = rows ? rows[r] : r;
        if (positions && positions[i] < 0) continue;        // padding token of a fixed-shape step
        const size_t at = (size_t)i * width, to = (size_t)r * width;
        if (y) {
            __syncthreads();                                 // the row before is through with these
            if (threadIdx.x < p.top) {
                s_place[threadIdx.x] = __ldcg(p.place + (size_t)i * p.top + threadIdx.x);
                s_weight[threadIdx.x] = __ldcg(p.weights + (size_t)i * p.top + threadIdx.x);
            }
            if (threadIdx.x == blockDim.x - 1)
                s_identity = h ? moe_identity_weight(p.experts, p.weights, i, p.top, p.n_real) : 0.f;
        }
        float ss = 0.f;
        if constexpr (VPT > 0) {
            float4 v[VPT];
#pragma unroll
            for (int j = 0; j < VPT; ++j) {
                const int c = 4 * (threadIdx.x + j * blockDim.x);
                v[j] = make_float4(0.f, 0.f, 0.f, 0.f);
                if (c >= width) continue;
                v[j] = load4_cg(x + at + c);
                if (p.e) v[j] = add4(v[j], load4_cg(p.e + at + c));
            }
            if (y) __syncthreads();
#pragma unroll
            for (int j = 0; j < VPT; ++j) {
                const int c = 4 * (threadIdx.x + j * blockDim.x);
                if (c >= width) continue;
                float4 u = make_float4(0.f, 0.f, 0.f, 0.f), d = u;
                if (p.f) u = load4_cg(p.f + at + c);
                if (y) {
#pragma unroll 4
                    for (int k = 0; k < p.top; ++k) {
                        const int pl = s_place[k];
                        if (pl < 0) continue;
                        const float w = s_weight[k];
                        const float4 q = load4_cg(y + (size_t)pl * width + c);
                        u = make_float4(fmaf(w, q.x, u.x), fmaf(w, q.y, u.y), fmaf(w, q.z, u.z), fmaf(w, q.w, u.w));
                    }
                    const float w = s_identity;
                    if (w != 0.f) {
                        const float4 q = load4_cg(h + at + c);
                        u = make_float4(fmaf(w, q.x, u.x), fmaf(w, q.y, u.y), fmaf(w, q.z, u.z), fmaf(w, q.w, u.w));
                    }
                }
                if (p.f || y) {
                    const float4 s = load4(p.s2 + c);
                    d = make_float4(s.x * u.x, s.y * u.y, s.z * u.z, s.w * u.w);
                }
                if (p.a) {
                    const float4 s = load4(p.s1 + c), q = load4_cg(p.a + at + c);
                    d = make_float4(fmaf(s.x, q.x, d.x), fmaf(s.y, q.y, d.y), fmaf(s.z, q.z, d.z), fmaf(s.w, q.w, d.w));
                }
                v[j] = add4(v[j], d);
                if (pending && !rows) store4(x + at + c, v[j]);
                ss += (v[j].x * v[j].x + v[j].y * v[j].y) + (v[j].z * v[j].z + v[j].w * v[j].w);
            }
            if (!out1 && !out2) continue;
            const float k = 1.f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
#pragma unroll
            for (int j = 0; j < VPT; ++j) {
                const int c = 4 * (threadIdx.x + j * blockDim.x);
                if (c >= width) continue;
                const float4 n = make_float4(v[j].x * k, v[j].y * k, v[j].z * k, v[j].w * k);
                if (out1) {
                    const float4 w = load4(w1 + c);
                    store4(out1 + to + c, make_float4(n.x * w.x, n.y * w.y, n.z * w.z, n.w * w.w));
                }
                if (out2) {
                    const float4 w = load4(w2 + c);
                    store4(out2 + to + c, make_float4(n.x * w.x, n.y * w.y, n.z * w.z, n.w * w.w));
                }
            }
        } else {
            if (y) __syncthreads();
            // (a thread reads back only what it wrote itself)
            for (int c = threadIdx.x; c < width; c += blockDim.x) {
                float v = __ldcg(x + at + c), u = 0.f, d = 0.f;
                if (p.e) v += __ldcg(p.e + at + c);
                if (p.f) u = __ldcg(p.f + at + c);
                if (y) {
                    for (int k = 0; k < p.top; ++k)
                        if (s_place[k] >= 0) u = fmaf(s_weight[k], load1_cg(y + (size_t)s_place[k] * width + c), u);
                    if (s_identity != 0.f) u = fmaf(s_identity, load1_cg(h + at + c), u);
                }
                if (p.f || y) d = p.s2[c] * u;
                if (p.a) d = fmaf(p.s1[c], __ldcg(p.a + at + c), d);
                v += d;
                if (pending && !rows) x[at + c] = v;
                sn_row[c] = v;
                ss = fmaf(v, v, ss);
            }
            if (!out1 && !out2) continue;
            const float k = 1.f / sqrtf(block_sum(ss, scratch) / (float)width + eps);
            for (int c = threadIdx.x; c < width; c += blockDim.x) {
                if (out1) out1[to + c] = from_f32<T>(sn_row[c] * k * w1[c]);
                if (out2) out2[to + c] = from_f32<T>(sn_row[c] * k * w2[c]);
            }
        }
    }
}

// The most choices per token whose experts' rows the kernel sums itself.
ST_EXPORT int st_scaled_sum_norms_max_top() { return SN_MAX_TOP; }

// dtype: the type of y, h, out1 and out2
ST_EXPORT int st_scaled_sum_norms(float* x, const float* a, const float* s1, const float* f, const float* s2, const float* e,
                                  const void* y, const int* place, const float* weights, const int* experts, int top,
                                  int n_real, const void* h, const float* w1, const float* w2, float eps, const int* rows,
                                  int n_rows, int width, const int* positions, void* out1, void* out2, int dtype,
                                  void* stream) {
    if (n_rows <= 0) return 0;
    if (width <= 0 || (a && !s1) || ((f || y) && !s2) || (f && y) || (out1 && !w1) || (out2 && !w2)) return ST_ERR_BAD_ARG;
    if (y && (!place || !weights || top <= 0 || (h && !experts))) return ST_ERR_BAD_ARG;
    if (y && top > SN_MAX_TOP) return ST_ERR_TOO_LARGE;
    if ((size_t)width * sizeof(float) > 200 * 1024) return ST_ERR_TOO_LARGE;
    const ScaledSum p{a, s1, f, s2, e, y, y ? h : nullptr, place, experts, weights, top, n_real};
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = width % 4 == 0 && width <= 8192 && aligned16(x) && aligned16(a) && aligned16(s1) && aligned16(f) &&
                     aligned16(s2) && aligned16(e) && aligned16(y) && aligned16(h) && aligned16(w1) && aligned16(w2) &&
                     aligned16(out1) && aligned16(out2);
    const int vpt = !vec ? 0 : width <= 2048 ? 1 : width <= 4096 ? 2 : 4;
    int block = vpt ? ((width + 4 * vpt - 1) / (4 * vpt) + 31) / 32 * 32 : 256;
    if (block < 64) block = 64;                              // a thread per choice
    if (block > 512) block = 512;
    const size_t smem = vpt ? 0 : (size_t)width * sizeof(float);
    int grid = st_sm_count() * 4;
    if (grid > n_rows) grid = n_rows;
#define SN_LAUNCH(T, VPT)                                                                                                 \
    do {                                                                                                                  \
        auto kern = scaled_sum_norms_kernel<T, VPT>;                                                                      \
        if (smem > 40 * 1024) {                                                                                           \
            cudaError_t err = cudaFuncSetAttribute(kern, cudaFuncAttributeMaxDynamicSharedMemorySize, (int)smem);         \
            if (err != cudaSuccess) return (int)err;                                                                      \
        }                                                                                                                 \
        return st_launch_pdl("scaled_sum_norms", kern, dim3(grid), dim3(block), smem, s, x, p, w1, w2, eps, rows, n_rows, \
                             width, positions, (T*)out1, (T*)out2);                                                       \
    } while (0)
#define SN_PICK(T)                          \
    do {                                    \
        if (vpt == 0) SN_LAUNCH(T, 0);      \
        if (vpt == 1) SN_LAUNCH(T, 1);      \
        if (vpt == 2) SN_LAUNCH(T, 2);      \
        SN_LAUNCH(T, 4);                    \
    } while (0)
    if (dtype == 0) SN_PICK(float);
    if (dtype != 1) return ST_ERR_BAD_DTYPE;
    SN_PICK(bf16);
#undef SN_PICK
#undef SN_LAUNCH
}
