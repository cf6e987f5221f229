// The selective scan: a diagonal recurrence whose decay, write strength and read-out are made from the token itself.
//
// Per channel c and state element n, with d_c = softplus(r_c + b_c) the step size, A < 0 and token rows B, C shared by
// all channels:
//
//   S[c, n] <- exp(d_c A[c, n]) S[c, n] + d_c x_c B_n        y_c = sum_n S[c, n] C_n + D_c x_c
//   out_c   =  y_c * silu(z_c)
//
// S is float and lives in a state slot per request; everything from the step sizes on is float arithmetic.
//
// A thread owns NS state elements of one channel (lpc lanes share a channel when the state is longer) and walks its
// tokens; the rows B and C of 4 to 32 tokens at a time stand in shared memory.
//
// mamba_scan with chunks (long portions): the recurrence is linear in S, and the product of a run of decays is
// exp(A * sum of step sizes).  The tokens of every request are cut into chunks of `chunk` tokens (a list of (request,
// offset) made on the host):
//   local    every chunk but a request's last is scanned from a zero state: its end state and the sum of its steps
//   combine  per state element, the chunks of a request in order: the true state each chunk starts from
//   final    every chunk scanned from its true state; a request's last chunk leaves the request's new state
// so the serial chain is `chunk` tokens long instead of the whole portion.  Step sizes are finished (bias, softplus) in
// place by the local pass; a request's last chunk finishes its own.
// mamba_scan without chunks (short portions): the final pass alone, one item per request, from the state slot.
// mamba_single (every request brings one token): the low-rank product that gives r_c happens in the kernel too, and
// four elements per thread spread the state over more threads.
//
// For float storage the exponentials are expf; for bfloat16 they are ex2.approx with A scaled by log2(e).
#include "common.cuh"

#define MS_THREADS 128
#define MS_AHEAD 4          // tokens whose inputs are asked for together

__device__ __forceinline__ float ms_softplus(float v) { return v > 20.f ? v : log1pf(expf(v)); }
template <typename T> __device__ __forceinline__ float ms_decay(float e);
template <> __device__ __forceinline__ float ms_decay<float>(float e) { return expf(e); }
template <> __device__ __forceinline__ float ms_decay<bf16>(float e) {
    float y;
    asm("ex2.approx.ftz.f32 %0, %1;\n" : "=f"(y) : "f"(e));
    return y;
}
template <typename T> __device__ __forceinline__ float ms_unit();       // what A is multiplied by for ms_decay
template <> __device__ __forceinline__ float ms_unit<float>() { return 1.f; }
template <> __device__ __forceinline__ float ms_unit<bf16>() { return 1.4426950408889634f; }

template <typename T>
struct ScanArgs {
    const T* x;                 // [tokens, inner]
    float* dt;                  // [tokens, inner]: step logits without the bias; finished in place by the local pass
    const float* xd;            // [tokens, xd_ld]: B at b_off, C at c_off
    int xd_ld, b_off, c_off;
    const T* z;                 // [tokens, z_ld]
    int z_ld;
    T* out;                     // [tokens, inner]
    const float *A, *D, *dt_b;  // [inner, n], [inner], [inner]
    float* state;               // [slots, inner, n]
    float* buf;                 // [chunks, inner, n]: end states of the local pass, then start states
    float* sums;                // [chunks, inner]: sums of step sizes
    const int *positions, *q_start, *slots, *chunks, *chunk_first;
    int inner, n, lpc, chunk, tile, write_state;
};

template <int NS>
__device__ __forceinline__ void ms_load_row(const float* p, int first, int n, float* v) {
#pragma unroll
    for (int i = 0; i < NS; i += 4) {
        if (n % 4 == 0 && first + i < n) {
            const float4 q = __ldcg(reinterpret_cast<const float4*>(p + first + i));
            v[i] = q.x; v[i + 1] = q.y; v[i + 2] = q.z; v[i + 3] = q.w;
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j) v[i + j] = first + i + j < n ? __ldcg(p + first + i + j) : 0.f;
        }
    }
}
template <int NS>
__device__ __forceinline__ void ms_store_row(float* p, int first, int n, const float* v) {
#pragma unroll
    for (int i = 0; i < NS; i += 4) {
        if (n % 4 == 0 && first + i < n) {
            *reinterpret_cast<float4*>(p + first + i) = make_float4(v[i], v[i + 1], v[i + 2], v[i + 3]);
        } else {
#pragma unroll
            for (int j = 0; j < 4; ++j)
                if (first + i + j < n) p[first + i + j] = v[i + j];
        }
    }
}

// LOCAL: the scan from a zero state that leaves end state and sum of steps; otherwise the scan that leaves outputs
template <typename T, int NS, bool LOCAL>
__global__ void __launch_bounds__(MS_THREADS, NS <= 16 ? 7 : 4)
mamba_scan_kernel(ScanArgs<T> a) {
    extern __shared__ __align__(16) float ms_smem[];
    const int lpc = a.lpc, nsp = NS * lpc, per_block = MS_THREADS / lpc;
    float* sB = ms_smem;                        // [tile][nsp]
    float* sC = ms_smem + a.tile * nsp;         // [tile][nsp]
    const int part = threadIdx.x % lpc, ch = blockIdx.y * per_block + threadIdx.x / lpc;
    const bool on = ch < a.inner;
    float A[NS], S[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) {              // (a state element beyond n decays by exp(0) and stays zero)
        const int e = part * NS + i;
        A[i] = (on && e < a.n) ? a.A[(size_t)ch * a.n + e] * ms_unit<T>() : 0.f;
    }
    const float bias = on ? a.dt_b[ch] : 0.f, Dc = (on && !LOCAL) ? a.D[ch] : 0.f;
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    int req = blockIdx.x, off = 0;
    if (a.chunks) {
        req = a.chunks[2 * blockIdx.x];
        off = a.chunks[2 * blockIdx.x + 1];
    }
    const int first = a.q_start[req], n_new = a.q_start[req + 1] - first;
    if (off >= n_new || a.positions[first] < 0) return;         // padding: a chunk, a request, or a token at -1
    const bool last = !a.chunks || off + a.chunk >= n_new;
    if (LOCAL && last) return;
    const int t0 = first + off, count = a.chunks ? min(a.chunk, n_new - off) : n_new;
    const bool raw = LOCAL || last;                             // the step sizes still are logits
    float* slot = a.state + ((size_t)a.slots[req] * a.inner + (on ? ch : 0)) * a.n;
    float* cell = a.chunks ? a.buf + ((size_t)blockIdx.x * a.inner + (on ? ch : 0)) * a.n : slot;
#pragma unroll
    for (int i = 0; i < NS; ++i) S[i] = 0.f;
    if (!LOCAL && on) ms_load_row<NS>(cell, part * NS, a.n, S);
    float total = 0.f;
    for (int base = 0; base < count; base += a.tile) {
        const int m = min(a.tile, count - base);
        __syncthreads();
        for (int i = threadIdx.x; i < m * nsp; i += MS_THREADS) {
            const int r = i / nsp, e = i % nsp;
            const float* row = a.xd + (size_t)(t0 + base + r) * a.xd_ld;
            sB[i] = e < a.n ? __ldcg(row + a.b_off + e) : 0.f;
            if (!LOCAL) sC[i] = e < a.n ? __ldcg(row + a.c_off + e) : 0.f;
        }
        __syncthreads();
        for (int k0 = 0; k0 < m; k0 += MS_AHEAD) {
            float xv[MS_AHEAD], dv[MS_AHEAD], zv[MS_AHEAD];
#pragma unroll
            for (int u = 0; u < MS_AHEAD; ++u) {
                xv[u] = dv[u] = zv[u] = 0.f;
                if (!on || k0 + u >= m) continue;
                const size_t t = (size_t)(t0 + base + k0 + u);
                xv[u] = load1_cg(a.x + t * a.inner + ch);
                dv[u] = __ldcg(a.dt + t * a.inner + ch);
                if (!LOCAL) zv[u] = load1_cg(a.z + t * a.z_ld + ch);
            }
#pragma unroll
            for (int u = 0; u < MS_AHEAD; ++u) {
                if (k0 + u >= m) break;                          // (the same for the whole block)
                const size_t t = (size_t)(t0 + base + k0 + u);
                const float d = raw ? ms_softplus(dv[u] + bias) : dv[u];
                const float dx = d * xv[u];
                const float4* b4 = reinterpret_cast<const float4*>(sB + (k0 + u) * nsp + part * NS);
                const float4* c4 = reinterpret_cast<const float4*>(sC + (k0 + u) * nsp + part * NS);
                float y0 = 0.f, y1 = 0.f, y2 = 0.f, y3 = 0.f;
#pragma unroll
                for (int i = 0; i < NS / 4; ++i) {
                    const float4 b = b4[i];
                    S[4 * i] = fmaf(ms_decay<T>(d * A[4 * i]), S[4 * i], dx * b.x);
                    S[4 * i + 1] = fmaf(ms_decay<T>(d * A[4 * i + 1]), S[4 * i + 1], dx * b.y);
                    S[4 * i + 2] = fmaf(ms_decay<T>(d * A[4 * i + 2]), S[4 * i + 2], dx * b.z);
                    S[4 * i + 3] = fmaf(ms_decay<T>(d * A[4 * i + 3]), S[4 * i + 3], dx * b.w);
                    if (!LOCAL) {
                        const float4 c = c4[i];
                        y0 = fmaf(S[4 * i], c.x, y0);
                        y1 = fmaf(S[4 * i + 1], c.y, y1);
                        y2 = fmaf(S[4 * i + 2], c.z, y2);
                        y3 = fmaf(S[4 * i + 3], c.w, y3);
                    }
                }
                if (LOCAL) {
                    total += d;
                    if (on && part == 0) a.dt[t * a.inner + ch] = d;
                } else {
                    float y = (y0 + y1) + (y2 + y3);
                    for (int o = lpc >> 1; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
                    if (on && part == 0) {
                        y = fmaf(Dc, xv[u], y);
                        a.out[t * a.inner + ch] = from_f32<T>(y * (zv[u] / (1.f + expf(-zv[u]))));
                    }
                }
            }
        }
    }
    if (!on) return;
    if (LOCAL) {
        ms_store_row<NS>(cell, part * NS, a.n, S);
        if (part == 0) a.sums[(size_t)blockIdx.x * a.inner + ch] = total;
    } else if (last && a.write_state) {
        ms_store_row<NS>(slot, part * NS, a.n, S);
    }
}

// buf[k] (the end state of chunk k from zero) <- the state chunk k starts from, for the chunks of every request in order
#define MC_AHEAD 4
__global__ void __launch_bounds__(256)
mamba_combine_kernel(float* __restrict__ buf, const float* __restrict__ sums, const float* __restrict__ A,
                     const float* __restrict__ state, const int* __restrict__ positions, const int* __restrict__ q_start,
                     const int* __restrict__ slots, const int* __restrict__ chunk_first, int inner, int n) {
    const size_t per = (size_t)inner * n, e = (size_t)blockIdx.x * blockDim.x + threadIdx.x;
    const float Ae = e < per ? A[e] : 0.f;
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    const int req = blockIdx.y;
    const int first = q_start[req];
    if (e >= per || q_start[req + 1] <= first || positions[first] < 0) return;
    const int k0 = chunk_first[req], k1 = chunk_first[req + 1];
    const int ch = (int)(e / n);
    float S = __ldcg(state + (size_t)slots[req] * per + e);
    for (int k = k0; k < k1; k += MC_AHEAD) {
        float loc[MC_AHEAD], sd[MC_AHEAD];
#pragma unroll
        for (int u = 0; u < MC_AHEAD; ++u) {                     // (the last chunk has no end state: nothing reads what follows it)
            const bool has = k + u + 1 < k1;
            loc[u] = has ? __ldcg(buf + (size_t)(k + u) * per + e) : 0.f;
            sd[u] = has ? __ldcg(sums + (size_t)(k + u) * inner + ch) : 0.f;
        }
#pragma unroll
        for (int u = 0; u < MC_AHEAD; ++u) {
            if (k + u >= k1) break;
            buf[(size_t)(k + u) * per + e] = S;
            S = fmaf(expf(Ae * sd[u]), S, loc[u]);
        }
    }
}

static int ms_lanes(int n, int ns) {            // lanes per channel: a power of two
    int lpc = 1;
    while (lpc * ns < n) lpc *= 2;
    return lpc;
}

template <typename T, int NS>
static int launch_scan(ScanArgs<T> a, int n_seqs, int n_chunks, cudaStream_t s) {
    a.lpc = ms_lanes(a.n, NS);
    const int nsp = NS * a.lpc, per_block = MS_THREADS / a.lpc, ny = (a.inner + per_block - 1) / per_block;
    a.tile = nsp <= 128 ? 32 : 4096 / nsp;
    const size_t smem = 2 * (size_t)a.tile * nsp * sizeof(float);
    if (a.chunks) {
        int rc = st_launch_pdl("mamba_local", mamba_scan_kernel<T, NS, true>, dim3(n_chunks, ny), dim3(MS_THREADS), smem, s, a);
        if (rc) return rc;
        const size_t per = (size_t)a.inner * a.n;
        rc = st_launch_pdl("mamba_combine", mamba_combine_kernel, dim3((unsigned)((per + 255) / 256), n_seqs), dim3(256), 0, s, a.buf,
                           (const float*)a.sums, a.A, (const float*)a.state, a.positions, a.q_start, a.slots, a.chunk_first,
                           a.inner, a.n);
        if (rc) return rc;
        return st_launch_pdl("mamba_scan", mamba_scan_kernel<T, NS, false>, dim3(n_chunks, ny), dim3(MS_THREADS), smem, s, a);
    }
    return st_launch_pdl("mamba_scan", mamba_scan_kernel<T, NS, false>, dim3(n_seqs, ny), dim3(MS_THREADS), smem, s, a);
}

// chunks: int32 [n_chunks][2] = (request of the step, offset of the chunk among its new tokens), the chunks of a request
// side by side and in order, offsets past a request's tokens: padding; chunk_first [n_seqs + 1]: where each request's
// chunks begin; buf float [n_chunks, inner, n], sums float [n_chunks, inner].  Null: no chunks.
ST_EXPORT int st_mamba_scan(const void* x, float* dt, const float* xd, int xd_ld, int b_off, int c_off, const void* z,
                            int z_ld, void* out, const float* A, const float* D, const float* dt_b, float* state,
                            int write_state, float* buf, float* sums, const int* positions, const int* q_start,
                            const int* slots, int n_seqs, const int* chunks, const int* chunk_first, int n_chunks,
                            int chunk, int inner, int n, int dtype, void* stream) {
    if (n_seqs <= 0) return 0;
    if (inner <= 0 || n <= 0 || b_off < 0 || c_off < 0 || b_off + n > xd_ld || c_off + n > xd_ld || z_ld < inner) return ST_ERR_BAD_ARG;
    if (chunks && (chunk <= 0 || n_chunks <= 0 || !buf || !sums || !chunk_first)) return ST_ERR_BAD_ARG;
    if (n > 1024 || n_seqs > 65535) return ST_ERR_TOO_LARGE;
    cudaStream_t s = (cudaStream_t)stream;
#define MS_ARGS(T)                                                                                                       \
    ScanArgs<T> a{(const T*)x, dt, xd, xd_ld, b_off, c_off, (const T*)z, z_ld, (T*)out, A, D, dt_b, state, buf, sums,    \
                  positions, q_start, slots, chunks, chunk_first, inner, n, 1, chunk, 32, write_state}
#define MS_PICK(T)                                                   \
    do {                                                             \
        MS_ARGS(T);                                                  \
        if (n <= 4) return launch_scan<T, 4>(a, n_seqs, n_chunks, s);   \
        if (n <= 8) return launch_scan<T, 8>(a, n_seqs, n_chunks, s);   \
        if (n <= 16) return launch_scan<T, 16>(a, n_seqs, n_chunks, s); \
        return launch_scan<T, 32>(a, n_seqs, n_chunks, s);           \
    } while (0)
    if (dtype == 0) MS_PICK(float);
    if (dtype == 1) MS_PICK(bf16);
    return ST_ERR_BAD_DTYPE;
#undef MS_PICK
}

// ------------------------------------------------------------------------------------------------
// eight neighbouring weights times eight floats
__device__ __forceinline__ float ms_dot8(const float* w, const float* v, float acc) {
    const float4 p = load4(w), q = load4(w + 4), a = load4(v), b = load4(v + 4);
    acc = fmaf(p.x, a.x, fmaf(p.y, a.y, fmaf(p.z, a.z, fmaf(p.w, a.w, acc))));
    return fmaf(q.x, b.x, fmaf(q.y, b.y, fmaf(q.z, b.z, fmaf(q.w, b.w, acc))));
}
__device__ __forceinline__ float ms_dot8(const bf16* w, const float* v, float acc) {
    const uint4 p = *reinterpret_cast<const uint4*>(w);
    const float4 a = load4(v), b = load4(v + 4);
    acc = fmaf(__uint_as_float(p.x << 16), a.x, fmaf(__uint_as_float(p.x & 0xffff0000u), a.y, acc));
    acc = fmaf(__uint_as_float(p.y << 16), a.z, fmaf(__uint_as_float(p.y & 0xffff0000u), a.w, acc));
    acc = fmaf(__uint_as_float(p.z << 16), b.x, fmaf(__uint_as_float(p.z & 0xffff0000u), b.y, acc));
    return fmaf(__uint_as_float(p.w << 16), b.z, fmaf(__uint_as_float(p.w & 0xffff0000u), b.w, acc));
}

template <typename T, int NS>
__global__ void __launch_bounds__(MS_THREADS)
mamba_single_kernel(const T* __restrict__ x, const float* __restrict__ xd, int xd_ld, int rank, int b_off, int c_off,
                    const T* __restrict__ w_dt, const T* __restrict__ z, int z_ld, T* __restrict__ out,
                    const float* __restrict__ A_, const float* __restrict__ D, const float* __restrict__ dt_b,
                    float* __restrict__ state, int write_state, const int* __restrict__ positions,
                    const int* __restrict__ seq_of_token, const int* __restrict__ slots, int inner, int n, int lpc) {
    extern __shared__ __align__(16) float ms_smem[];
    const int nsp = NS * lpc, per_block = MS_THREADS / lpc;
    float* sR = ms_smem;                        // [rank] inputs of the low-rank product
    float* sB = sR + rank;                      // [nsp]
    float* sC = sB + nsp;                       // [nsp]
    const int part = threadIdx.x % lpc, ch = blockIdx.y * per_block + threadIdx.x / lpc;
    const bool on = ch < inner;
    float A[NS], S[NS];
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        const int e = part * NS + i;
        A[i] = (on && e < n) ? A_[(size_t)ch * n + e] * ms_unit<T>() : 0.f;
    }
    const float bias = on ? dt_b[ch] : 0.f, Dc = on ? D[ch] : 0.f;
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    const int t = blockIdx.x;
    if (positions[t] < 0) return;
    float* cell = state + ((size_t)slots[seq_of_token[t]] * inner + (on ? ch : 0)) * n;
#pragma unroll
    for (int i = 0; i < NS; ++i) S[i] = 0.f;
    if (on) ms_load_row<NS>(cell, part * NS, n, S);
    const float xv = on ? load1_cg(x + (size_t)t * inner + ch) : 0.f, zv = on ? load1_cg(z + (size_t)t * z_ld + ch) : 0.f;
    const float* row = xd + (size_t)t * xd_ld;
    for (int i = threadIdx.x; i < rank; i += MS_THREADS) sR[i] = __ldcg(row + i);
    for (int i = threadIdx.x; i < nsp; i += MS_THREADS) {
        sB[i] = i < n ? __ldcg(row + b_off + i) : 0.f;
        sC[i] = i < n ? __ldcg(row + c_off + i) : 0.f;
    }
    __syncthreads();
    float r = 0.f;
    if (on)
        for (int k = part * 8; k < rank; k += lpc * 8) r = ms_dot8(w_dt + (size_t)ch * rank + k, sR + k, r);
    for (int o = lpc >> 1; o > 0; o >>= 1) r += __shfl_xor_sync(0xffffffffu, r, o);
    const float d = ms_softplus(r + bias), dx = d * xv;
    float y = 0.f;
#pragma unroll
    for (int i = 0; i < NS; ++i) {
        S[i] = fmaf(ms_decay<T>(d * A[i]), S[i], dx * sB[part * NS + i]);
        y = fmaf(S[i], sC[part * NS + i], y);
    }
    for (int o = lpc >> 1; o > 0; o >>= 1) y += __shfl_xor_sync(0xffffffffu, y, o);
    if (!on) return;
    if (part == 0) out[(size_t)t * inner + ch] = from_f32<T>(fmaf(Dc, xv, y) * (zv / (1.f + expf(-zv))));
    if (write_state) ms_store_row<NS>(cell, part * NS, n, S);
}

// xd: [tokens, xd_ld] = low-rank inputs (`rank` of them, a multiple of 8) | ... B at b_off, C at c_off; w_dt [inner, rank]
ST_EXPORT int st_mamba_single(const void* x, const float* xd, int xd_ld, int rank, int b_off, int c_off, const void* w_dt,
                              const void* z, int z_ld, void* out, const float* A, const float* D, const float* dt_b,
                              float* state, int write_state, const int* positions, const int* seq_of_token,
                              const int* slots, int n_tokens, int inner, int n, int dtype, void* stream) {
    if (n_tokens <= 0) return 0;
    if (inner <= 0 || n <= 0 || rank <= 0 || rank % 8 || rank > xd_ld || b_off + n > xd_ld || c_off + n > xd_ld ||
        z_ld < inner || !aligned16(w_dt))
        return ST_ERR_BAD_ARG;
    if (n > 1024 || rank > 4096) return ST_ERR_TOO_LARGE;
    cudaStream_t s = (cudaStream_t)stream;
    const int ns = n <= 128 ? 4 : 32, lpc = ms_lanes(n, ns);
    const int per_block = MS_THREADS / lpc;
    const dim3 grid(n_tokens, (inner + per_block - 1) / per_block);
    const size_t smem = (size_t)(rank + 2 * ns * lpc) * sizeof(float);
#define M1_LAUNCH(T, NS)                                                                                               \
    return st_launch_pdl("mamba_single", mamba_single_kernel<T, NS>, grid, dim3(MS_THREADS), smem, s, (const T*)x, xd, xd_ld, rank, \
                         b_off, c_off, (const T*)w_dt, (const T*)z, z_ld, (T*)out, A, D, dt_b, state, write_state,     \
                         positions, seq_of_token, slots, inner, n, lpc)
    if (dtype == 0) { if (ns == 4) M1_LAUNCH(float, 4); M1_LAUNCH(float, 32); }
    if (dtype == 1) { if (ns == 4) M1_LAUNCH(bf16, 4); M1_LAUNCH(bf16, 32); }
    return ST_ERR_BAD_DTYPE;
#undef M1_LAUNCH
}
