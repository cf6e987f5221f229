// Routing of a mixture of experts: which experts a token uses, the tokens sorted by expert, and the weighted
// sum of the experts' results.
//
// moe_route:   z = W_r h (float, W_r float [experts, width]); s = softmax(z) over all experts; the `top` experts
//              with the largest s (ties: the lower index) and their s as weights (not renormalised, unless asked: then divided by their sum + 1e-20);
//              optionally g = sigmoid(w_g . h), one number per token (the gate of a shared expert).
//              RouteRule: scores may be sigmoid(z) instead; the experts may form equal groups of neighbours, of which
//              only the `keep` best (by the sum of a group's two largest scores; ties: the lower index) can be chosen
//              from; the weights are multiplied by `scale` in the end.  The logits may come from a product of their
//              own (z float [tokens, ld]) instead of being formed here.
//              With `correction` (float [experts]) experts, and groups, are chosen by s + correction, which may be
//              negative; the weights are the bare s.  group_max: a group counts by its largest choice score instead.
//              Which experts have weights of their own is not the router's business: outputs from n_real on may stand
//              for the identity (moe_sort gives them no place, moe_combine adds their weight times the input row).
//              A padding token (position < 0) gets expert -1.
// moe_sort:    the step's (token, choice) items grouped by expert: offsets[e]..offsets[e+1] are expert e's places
//              in `sorted` (item indices), `place[item]` the inverse, and a list of row tiles (expert, first place)
//              for the grouped products, padded with expert -1.  One block; items of one expert stand in no
//              particular order, which changes no result: every row of a product is computed on its own.
// moe_combine: out[t] = sum_k weight[t,k] * y[place[t,k]]  (+ g[t] * shared[t], or + shared[t] without gates), in float.
//              With identity experts: + h[t] times the sum of the weights whose expert is n_real or above.
#include "moe.cuh"

#define ROUTE_MAX_THREADS 1024     // a warp per router output up to this many
#define ROUTE_MAX_EXPERTS 1024

struct RouteRule {
    int sigmoid, groups, keep, renorm;      // groups <= 1: no groups
    float scale;
    const float* correction;                // added to the scores for the choice, or null
    int group_max;
};

// floats of shared memory a choice needs: scores, choice scores, group scores
__host__ __device__ __forceinline__ int route_floats(int n_experts, const RouteRule& rule) { return 2 * n_experts + rule.groups; }

// The choice of one token by one warp from its logits z[0..n_experts) in shared memory (overwritten).
__device__ __forceinline__ void route_choose(float* z, int n_experts, int top, const RouteRule& rule, int lane,
                                             int* __restrict__ experts, float* __restrict__ weights) {
    float inv = 1.f;
    if (rule.sigmoid) {
        for (int e = lane; e < n_experts; e += 32) z[e] = 1.f / (1.f + expf(-z[e]));
    } else {
        float m = -INFINITY;
        for (int e = lane; e < n_experts; e += 32) m = fmaxf(m, z[e]);
        m = warp_max(m);
        float sum = 0.f;
        for (int e = lane; e < n_experts; e += 32) {
            const float p = expf(z[e] - m);
            z[e] = p;
            sum += p;
        }
        inv = 1.f / warp_sum(sum);
    }
    __syncwarp();
    float* c = z + n_experts;              // what the choice goes by
    for (int e = lane; e < n_experts; e += 32) c[e] = rule.correction ? z[e] * inv + rule.correction[e] : z[e];
    __syncwarp();
    if (rule.groups > 1) {
        // a lane per group (in turns of 32): the sum of its two largest scores, or the largest; a group is kept
        // when fewer than `keep` groups stand before it (a larger value, or the same and a lower index)
        const int per = n_experts / rule.groups;
        float* gs = c + n_experts;
        for (int g = lane; g < rule.groups; g += 32) {
            float a = -INFINITY, b = -INFINITY;
            for (int i = 0; i < per; ++i) {
                const float v = c[g * per + i];
                if (v > a) { b = a; a = v; } else if (v > b) b = v;
            }
            gs[g] = per > 1 && !rule.group_max ? a + b : a;
        }
        __syncwarp();
        for (int g = lane; g < rule.groups; g += 32) {
            int before = 0;
            for (int o = 0; o < rule.groups; ++o) before += (gs[o] > gs[g] || (gs[o] == gs[g] && o < g)) ? 1 : 0;
            if (before >= rule.keep)
                for (int i = 0; i < per; ++i) c[g * per + i] = -INFINITY;
        }
        __syncwarp();
    }
    float chosen_sum = 0.f;
    for (int k = 0; k < top; ++k) {
        float best = -INFINITY;
        int arg = 0x7fffffff;
        for (int e = lane; e < n_experts; e += 32)
            if (c[e] > best) { best = c[e]; arg = e; }
#pragma unroll
        for (int o = 16; o > 0; o >>= 1) {
            const float ob = __shfl_xor_sync(0xffffffffu, best, o);
            const int oa = __shfl_xor_sync(0xffffffffu, arg, o);
            if (ob > best || (ob == best && oa < arg)) { best = ob; arg = oa; }
        }
        const bool any = arg < n_experts;            // (no expert is left in the kept groups: none, with weight 0)
        const float w = any ? z[arg] * inv : 0.f;
        chosen_sum += w;
        if (lane == 0) {
            experts[k] = any ? arg : -1;
            weights[k] = w * (rule.renorm ? 1.f : rule.scale);
            if (any) c[arg] = -INFINITY;
        }
        __syncwarp();
    }
    if (rule.renorm && lane == 0)
        for (int k = 0; k < top; ++k) weights[k] = weights[k] / (chosen_sum + 1e-20f) * rule.scale;
}

template <typename T>
__global__ void __launch_bounds__(ROUTE_MAX_THREADS)
moe_route_kernel(const T* __restrict__ h, int width, const float* __restrict__ w_r, int n_experts, int top,
                 RouteRule rule, const float* __restrict__ w_g, const int* __restrict__ positions,
                 int* __restrict__ experts, float* __restrict__ weights, float* __restrict__ gate, int vec) {
    extern __shared__ float z[];           // [route_floats + 1]
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    const int t = blockIdx.x;
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5, nwarp = blockDim.x / 32;
    if (positions && positions[t] < 0) {
        for (int k = threadIdx.x; k < top; k += blockDim.x) { experts[(size_t)t * top + k] = -1; weights[(size_t)t * top + k] = 0.f; }
        if (gate && threadIdx.x == 0) gate[t] = 0.f;
        return;
    }
    const T* row = h + (size_t)t * width;
    const int n_rows = n_experts + (w_g ? 1 : 0);
    for (int e = warp; e < n_rows; e += nwarp) {
        const float* wr = e < n_experts ? w_r + (size_t)e * width : w_g;
        float d = 0.f;
        if (vec) {
            // four at a time; a lane's partial sums run in the same order whatever the batch
#pragma unroll 8
            for (int i = lane * 4; i < width; i += 128) {
                const float4 a = load4_cg(row + i), c = *reinterpret_cast<const float4*>(wr + i);
                d = fmaf(a.x, c.x, fmaf(a.y, c.y, fmaf(a.z, c.z, fmaf(a.w, c.w, d))));
            }
        } else {
            for (int i = lane; i < width; i += 32) d = fmaf(load1_cg(row + i), wr[i], d);
        }
        d = warp_sum(d);
        if (lane == 0) z[e < n_experts ? e : route_floats(n_experts, rule)] = d;
    }
    __syncthreads();
    if (warp != 0) return;
    if (w_g && lane == 0) gate[t] = 1.f / (1.f + expf(-z[route_floats(n_experts, rule)]));
    route_choose(z, n_experts, top, rule, lane, experts + (size_t)t * top, weights + (size_t)t * top);
}

// The choice alone, from logits a product left: a warp per token.
#define CHOOSE_WARPS 4
__global__ void __launch_bounds__(CHOOSE_WARPS * 32)
moe_choose_kernel(const float* __restrict__ logits, int ld, int n_tokens, int n_experts, int top, RouteRule rule,
                  const int* __restrict__ positions, int* __restrict__ experts, float* __restrict__ weights) {
    extern __shared__ float z_all[];       // [CHOOSE_WARPS][route_floats]
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    const int lane = threadIdx.x & 31, warp = threadIdx.x >> 5;
    const int t = blockIdx.x * CHOOSE_WARPS + warp;
    if (t >= n_tokens) return;
    if (positions && positions[t] < 0) {
        for (int k = lane; k < top; k += 32) { experts[(size_t)t * top + k] = -1; weights[(size_t)t * top + k] = 0.f; }
        return;
    }
    float* z = z_all + warp * route_floats(n_experts, rule);
    for (int e = lane; e < n_experts; e += 32) z[e] = __ldcg(logits + (size_t)t * ld + e);
    __syncwarp();
    route_choose(z, n_experts, top, rule, lane, experts + (size_t)t * top, weights + (size_t)t * top);
}

static int route_rule_bad(const RouteRule& r, int n_experts, int top) {
    if (n_experts <= 0 || top <= 0 || top > n_experts || r.groups < 0) return 1;
    return r.groups > 1 && (n_experts % r.groups || r.keep <= 0 || r.keep > r.groups);
}

ST_EXPORT int st_moe_choose(const float* logits, int ld, int n_tokens, int n_experts, int top, int sigmoid, int groups,
                            int keep, int renorm, float scale, const float* correction, int group_max, const int* positions, int* experts,
                            float* weights, void* stream) {
    if (n_tokens <= 0) return 0;
    const RouteRule rule{sigmoid, groups, keep, renorm, scale, correction, group_max};
    if (route_rule_bad(rule, n_experts, top) || ld < n_experts) return ST_ERR_BAD_ARG;
    if (n_experts > ROUTE_MAX_EXPERTS) return ST_ERR_TOO_LARGE;
    const size_t smem = (size_t)CHOOSE_WARPS * route_floats(n_experts, rule) * sizeof(float);
    return st_launch_pdl("moe_choose", moe_choose_kernel, dim3((n_tokens + CHOOSE_WARPS - 1) / CHOOSE_WARPS), dim3(CHOOSE_WARPS * 32),
                         smem, (cudaStream_t)stream, logits, ld, n_tokens, n_experts, top, rule, positions, experts, weights);
}

ST_EXPORT int st_moe_route(const void* h, int n_tokens, int width, const float* w_r, int n_experts, int top, int sigmoid,
                           int groups, int keep, int renorm, float scale, const float* correction, int group_max, const float* w_g,
                           const int* positions, int* experts, float* weights, float* gate, int dtype, void* stream) {
    if (n_tokens <= 0) return 0;
    const RouteRule rule{sigmoid, groups, keep, renorm, scale, correction, group_max};
    if (route_rule_bad(rule, n_experts, top)) return ST_ERR_BAD_ARG;
    if (n_experts > ROUTE_MAX_EXPERTS) return ST_ERR_TOO_LARGE;
    cudaStream_t s = (cudaStream_t)stream;
    const size_t smem = (size_t)(route_floats(n_experts, rule) + 1) * sizeof(float);
    const int vec = width % 4 == 0 && aligned16(h) && aligned16(w_r) && (!w_g || aligned16(w_g));
    const int outputs = n_experts + (w_g ? 1 : 0);
    const int threads = outputs * 32 > ROUTE_MAX_THREADS ? ROUTE_MAX_THREADS : outputs * 32;
    if (dtype == 0)
        return st_launch_pdl("moe_route", moe_route_kernel<float>, dim3(n_tokens), dim3(threads), smem, s, (const float*)h,
                             width, w_r, n_experts, top, rule, w_g, positions, experts, weights, gate, vec);
    if (dtype == 1)
        return st_launch_pdl("moe_route", moe_route_kernel<bf16>, dim3(n_tokens), dim3(threads), smem, s, (const bf16*)h,
                             width, w_r, n_experts, top, rule, w_g, positions, experts, weights, gate, vec);
    return ST_ERR_BAD_DTYPE;
}

#define SORT_THREADS 1024

// offsets [n_experts + 1]; sorted [n_items]; place [n_items]; tile_group / tile_row0 [tile_cap]
__global__ void __launch_bounds__(SORT_THREADS)
moe_sort_kernel(const int* __restrict__ experts, int n_items, int n_experts, int tile_rows, int tile_cap,
                int* __restrict__ offsets, int* __restrict__ sorted, int* __restrict__ place,
                int* __restrict__ tile_group, int* __restrict__ tile_row0) {
    __shared__ int count[ROUTE_MAX_EXPERTS + 1];
    __shared__ int cursor[ROUTE_MAX_EXPERTS];
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    for (int e = threadIdx.x; e <= n_experts; e += SORT_THREADS) count[e] = 0;
    __syncthreads();
    for (int i = threadIdx.x; i < n_items; i += SORT_THREADS) {
        const int e = __ldcg(experts + i);
        if (e >= 0 && e < n_experts) atomicAdd(&count[e], 1);
    }
    __syncthreads();
    if (threadIdx.x == 0) {
        int run = 0, tile = 0;
        for (int e = 0; e < n_experts; ++e) {
            const int c = count[e];
            offsets[e] = run;
            cursor[e] = run;
            for (int r = 0; r < c && tile < tile_cap; r += tile_rows, ++tile) {
                tile_group[tile] = e;
                tile_row0[tile] = run + r;
            }
            run += c;
        }
        offsets[n_experts] = run;
        for (; tile < tile_cap; ++tile) { tile_group[tile] = -1; tile_row0[tile] = 0; }
    }
    __syncthreads();
    for (int i = threadIdx.x; i < n_items; i += SORT_THREADS) {
        const int e = __ldcg(experts + i);
        if (e >= 0 && e < n_experts) {
            const int p = atomicAdd(&cursor[e], 1);
            sorted[p] = i;
            place[i] = p;
        } else {
            place[i] = -1;
        }
    }
}

ST_EXPORT int st_moe_sort(const int* experts, int n_items, int n_experts, int tile_rows, int tile_cap, int* offsets,
                          int* sorted, int* place, int* tile_group, int* tile_row0, void* stream) {
    if (n_items <= 0) return 0;
    if (n_experts <= 0 || tile_rows <= 0) return ST_ERR_BAD_ARG;
    if (n_experts > ROUTE_MAX_EXPERTS) return ST_ERR_TOO_LARGE;
    if (tile_cap < (n_items + tile_rows - 1) / tile_rows + n_experts) return ST_ERR_BAD_SIZE;
    return st_launch_pdl("moe_sort", moe_sort_kernel, dim3(1), dim3(SORT_THREADS), 0, (cudaStream_t)stream, experts, n_items,
                         n_experts, tile_rows, tile_cap, offsets, sorted, place, tile_group, tile_row0);
}

template <typename T, typename TO, bool VEC>
__global__ void __launch_bounds__(256)
moe_combine_kernel(const T* __restrict__ y, const int* __restrict__ place, const float* __restrict__ weights, int top,
                   const T* __restrict__ shared, const float* __restrict__ gate, const int* __restrict__ experts, int n_real,
                   const T* __restrict__ h, int width, TO* __restrict__ out) {
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    const int t = blockIdx.x;
    const float w_id = h ? moe_identity_weight(experts, weights, t, top, n_real) : 0.f;
    if (VEC) {
        for (int e = threadIdx.x * 4; e < width; e += blockDim.x * 4) {
            float4 acc = make_float4(0.f, 0.f, 0.f, 0.f);
            for (int k = 0; k < top; ++k) {
                const int p = __ldcg(place + (size_t)t * top + k);
                if (p < 0) continue;
                const float w = __ldcg(weights + (size_t)t * top + k);
                const float4 v = load4_cg(y + (size_t)p * width + e);
                acc = make_float4(fmaf(w, v.x, acc.x), fmaf(w, v.y, acc.y), fmaf(w, v.z, acc.z), fmaf(w, v.w, acc.w));
            }
            if (shared) {
                const float w = gate ? __ldcg(gate + t) : 1.f;
                const float4 v = load4_cg(shared + (size_t)t * width + e);
                acc = make_float4(fmaf(w, v.x, acc.x), fmaf(w, v.y, acc.y), fmaf(w, v.z, acc.z), fmaf(w, v.w, acc.w));
            }
            if (w_id != 0.f) {
                const float4 v = load4_cg(h + (size_t)t * width + e);
                acc = make_float4(fmaf(w_id, v.x, acc.x), fmaf(w_id, v.y, acc.y), fmaf(w_id, v.z, acc.z), fmaf(w_id, v.w, acc.w));
            }
            store4(out + (size_t)t * width + e, acc);
        }
    } else
    for (int e = threadIdx.x; e < width; e += blockDim.x) {
        float acc = 0.f;
        for (int k = 0; k < top; ++k) {
            const int p = __ldcg(place + (size_t)t * top + k);
            if (p >= 0) acc = fmaf(__ldcg(weights + (size_t)t * top + k), load1_cg(y + (size_t)p * width + e), acc);
        }
        if (shared) acc = fmaf(gate ? __ldcg(gate + t) : 1.f, load1_cg(shared + (size_t)t * width + e), acc);
        if (w_id != 0.f) acc = fmaf(w_id, load1_cg(h + (size_t)t * width + e), acc);
        out[(size_t)t * width + e] = from_f32<TO>(acc);
    }
}

ST_EXPORT int st_moe_combine(const void* y, const int* place, const float* weights, int top, const void* shared,
                             const float* gate, const int* experts, int n_real, const void* h, int n_tokens, int width, void* out,
                             int dtype, int out_f32, void* stream) {
    if (n_tokens <= 0) return 0;
    if (h && !experts) return ST_ERR_BAD_ARG;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = width % 4 == 0 && aligned16(y) && aligned16(out) && aligned16(shared) && aligned16(h);
    int block = ((vec ? width / 4 : width) + 31) / 32 * 32;
    if (block > 256) block = 256;
#define MC_LAUNCH(T, TO, VEC)                                                                                           \
    return st_launch_pdl("moe_combine", moe_combine_kernel<T, TO, VEC>, dim3(n_tokens), dim3(block), 0, s, (const T*)y, \
                         place, weights, top, (const T*)shared, gate, experts, n_real, (const T*)h, width, (TO*)out)
    if (dtype == 0) {
        if (vec) MC_LAUNCH(float, float, true);
        MC_LAUNCH(float, float, false);
    }
    if (dtype != 1) return ST_ERR_BAD_DTYPE;
    if (out_f32) {
        if (vec) MC_LAUNCH(bf16, float, true);
        MC_LAUNCH(bf16, float, false);
    }
    if (vec) MC_LAUNCH(bf16, bf16, true);
    MC_LAUNCH(bf16, bf16, false);
#undef MC_LAUNCH
}
