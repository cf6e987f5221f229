// Short causal convolutions over time, one filter per channel, with the last
// taps-1 inputs of every request kept in a state slot so that a request may
// arrive in portions cut anywhere.
//
//   y[t][c] = sum_j w[c][j] * u[t - taps + 1 + j][c]          (zeros before position 0)
//
// conv_residual: out = u + y (or y alone).  conv_act: out = act(y + b) from the first columns of a wider projection,
// for mixers whose convolution stands inside.
//
// The state of a request holds the inputs at positions len-(taps-1) .. len-1
// in that order (zero where the position is negative: a fresh slot is all
// zeros, which is exactly "nothing before the sequence's start").
//
// Who may touch the state: within one launch the tokens of a request read the
// old state while its new state has to be written.  `conv_residual` gives the
// first token of a request in the step to the thread that also owns the
// request's state for that channel: it computes the outputs of the first
// taps-1 tokens itself (the only ones that read the state) and then writes the
// new state; all other threads read the step's own rows only.  A kernel that
// reads the state in many threads (the fused q/k/v preparation of
// diff_attention.cu) leaves it unchanged and is followed by
// `conv_state_update`, where one thread per (request, channel) reads all it
// needs before it writes.
#include "common.cuh"
#include <type_traits>

#define CONV_MAX_TAPS 8

template <int V, typename T> __device__ __forceinline__ void load_v(const T* p, float* v) {
    // through L2 only: the rows were written by the kernel just before (see the note on programmatic launch)
    if (V == 4) { const float4 f = load4_cg(p); v[0] = f.x; v[1] = f.y; v[2] = f.z; v[3] = f.w; }
    else v[0] = load1_cg(p);
}
template <int V, typename T> __device__ __forceinline__ void store_v(T* p, const float* v) {
    if (V == 4) store4(p, make_float4(v[0], v[1], v[2], v[3]));
    else p[0] = from_f32<T>(v[0]);
}

// out[t][c] = (residual ? in[t][c] : 0) + conv(in)[t][c];  in: float residual rows or activations.
// A thread owns V neighbouring channels (V = 4: 16-byte accesses, channels % 4 == 0).
template <typename TI, typename TO, int V>
__global__ void __launch_bounds__(128)
conv_residual_kernel(const TI* __restrict__ in, const float* __restrict__ w, float* __restrict__ state,
                     TO* __restrict__ out, const int* __restrict__ positions, const int* __restrict__ seq_of_token,
                     const int* __restrict__ q_start, const int* __restrict__ slots, int channels, int taps,
                     int residual) {
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    const int t = blockIdx.x;
    float wv[V][CONV_MAX_TAPS];
    if (c < channels) {                                 // the filters: no kernel writes them, fetched before the wait
#pragma unroll
        for (int v = 0; v < V; ++v)
#pragma unroll
            for (int j = 0; j < CONV_MAX_TAPS; ++j)     // (constant bounds: the filters stay in registers)
                wv[v][j] = j < taps ? w[(size_t)(c + v) * taps + j] : 0.f;
    }
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    if (c >= channels || positions[t] < 0) return;      // padding token of a fixed-shape step
    const int b = seq_of_token[t];
    const int first = q_start[b], n = q_start[b + 1] - first, i = t - first;
    const int keep = taps - 1;
    if (i >= keep) {
        float y[V], x[V];
#pragma unroll
        for (int v = 0; v < V; ++v) y[v] = 0.f;
#pragma unroll
        for (int j = 0; j < CONV_MAX_TAPS; ++j) {
            if (j < taps) {
                load_v<V>(in + (size_t)(t - keep + j) * channels + c, x);
#pragma unroll
                for (int v = 0; v < V; ++v) y[v] = fmaf(wv[v][j], x[v], y[v]);
            }
        }
#pragma unroll
        for (int v = 0; v < V; ++v) y[v] += residual ? x[v] : 0.f;      // x holds the token's own row (j = taps - 1)
        store_v<V>(out + (size_t)t * channels + c, y);
        return;
    }
    if (i != 0) return;                                 // done by the thread of the request's first token
    // u = old state followed by the first rows of the step: u[keep + k] is the step's token k
    float* st = state + (size_t)slots[b] * keep * channels + c;
    float u[2 * CONV_MAX_TAPS][V];
    const int m = n < keep ? n : keep;                  // tokens that read the state
    for (int j = 0; j < keep; ++j) load_v<V>(st + (size_t)j * channels, u[j]);
    for (int k = 0; k < m; ++k) load_v<V>(in + (size_t)(first + k) * channels + c, u[keep + k]);
    for (int k = 0; k < m; ++k) {
        float y[V];
#pragma unroll
        for (int v = 0; v < V; ++v) {
            y[v] = 0.f;      // (the filters once more from memory: indexing wv by a variable would move it out of registers)
            for (int j = 0; j < taps; ++j) y[v] = fmaf(w[(size_t)(c + v) * taps + j], u[k + j][v], y[v]);
            y[v] += residual ? u[keep + k][v] : 0.f;
        }
        store_v<V>(out + (size_t)(first + k) * channels + c, y);
    }
    // the last `keep` inputs of old state + all n rows
    for (int j = 0; j < keep; ++j) {
        const int src = n + j;                          // index into (state, rows of the step)
        float x[V];
        if (src < keep) {
#pragma unroll
            for (int v = 0; v < V; ++v) x[v] = u[src][v];
        } else {
            load_v<V>(in + (size_t)(first + src - keep) * channels + c, x);
        }
        store_v<V>(st + (size_t)j * channels, x);
    }
}

// state <- the last taps-1 rows of (state, the request's rows of this step), for every request of the step
template <typename TI>
__global__ void __launch_bounds__(256)
conv_state_update_kernel(const TI* __restrict__ in, int ld, float* __restrict__ state,
                         const int* __restrict__ positions, const int* __restrict__ q_start,
                         const int* __restrict__ slots, int channels, int taps) {
    const int c = blockIdx.x * blockDim.x + threadIdx.x;
    const int b = blockIdx.y;
    const int first = q_start[b], n = q_start[b + 1] - first;
    // padding of a fixed-shape step: a request without tokens, or one whose tokens stand at position -1
    if (c >= channels || n <= 0 || positions[first] < 0) return;
    const int keep = taps - 1;
    float* st = state + (size_t)slots[b] * keep * channels + c;
    float v[CONV_MAX_TAPS];
    for (int j = 0; j < keep; ++j) {
        const int src = n + j;
        v[j] = src < keep ? st[(size_t)src * channels] : to_f32(in[(size_t)(first + src - keep) * ld + c]);
    }
    for (int j = 0; j < keep; ++j) st[(size_t)j * channels] = v[j];
}

// V neighbouring inputs as they stand in memory (asked for early, widened when they are used)
template <typename T, int V> struct ConvRaw;
template <> struct ConvRaw<float, 1> {
    float r;
    __device__ __forceinline__ void load(const float* p) { r = __ldcg(p); }
    __device__ __forceinline__ void widen(float* v) const { v[0] = r; }
};
template <> struct ConvRaw<bf16, 1> {
    unsigned short r;
    __device__ __forceinline__ void load(const bf16* p) { r = __ldcg(reinterpret_cast<const unsigned short*>(p)); }
    __device__ __forceinline__ void widen(float* v) const { v[0] = __uint_as_float((unsigned)r << 16); }
};
template <> struct ConvRaw<float, 4> {
    float4 r;
    __device__ __forceinline__ void load(const float* p) { r = __ldcg(reinterpret_cast<const float4*>(p)); }
    __device__ __forceinline__ void widen(float* v) const { v[0] = r.x; v[1] = r.y; v[2] = r.z; v[3] = r.w; }
};
template <> struct ConvRaw<bf16, 4> {
    uint2 r;
    __device__ __forceinline__ void load(const bf16* p) { r = __ldcg(reinterpret_cast<const uint2*>(p)); }
    __device__ __forceinline__ void widen(float* v) const {
        v[0] = __uint_as_float(r.x << 16); v[1] = __uint_as_float(r.x & 0xffff0000u);
        v[2] = __uint_as_float(r.y << 16); v[3] = __uint_as_float(r.y & 0xffff0000u);
    }
};

// out[t][c] = act(bias[c] + conv(in)[t][c]);  in: [tokens, ld], its first `channels` columns.  A thread owns V
// neighbouring channels of TT consecutive tokens of the step: its tokens' rows and the K - 1 rows before the first are
// asked for at once (K: the number of taps, rounded up to 4 or 8; the taps that are not there have weight zero).  Rows
// from before the step come from the request's state.  Where the thread's tokens belong to several requests it takes
// them one by one.  The state is read by several threads and stays as it is (conv_state_update follows), unless
// `move_state` says that every request brings exactly one token: then the one thread that reads a request's state for
// a channel also moves it on.
template <typename T, int V, int TT, int K>
__global__ void __launch_bounds__(128)
conv_act_kernel(const T* __restrict__ in, int ld, const float* __restrict__ w, const float* __restrict__ bias,
                float* __restrict__ state, T* __restrict__ out, const int* __restrict__ positions,
                const int* __restrict__ seq_of_token, const int* __restrict__ q_start, const int* __restrict__ slots,
                int n_tokens, int channels, int taps, int act, int move_state) {
    const int c = (blockIdx.y * blockDim.x + threadIdx.x) * V;
    float wv[V][K], bv[V];
    if (c < channels) {                                 // no kernel writes the filters: fetched before the wait
#pragma unroll
        for (int v = 0; v < V; ++v) {
            bv[v] = bias ? bias[c + v] : 0.f;
            if (taps == 4 && K == 4) {                  // (a channel's filter is one 16-byte piece)
                const float4 q = load4(w + (size_t)(c + v) * 4);
                wv[v][0] = q.x; wv[v][1] = q.y; wv[v][2] = q.z; wv[v][3] = q.w;
                continue;
            }
#pragma unroll
            for (int j = 0; j < K; ++j)                 // the newest input's weight stands last, whatever taps is
                wv[v][j] = j >= K - taps ? w[(size_t)(c + v) * taps + j - (K - taps)] : 0.f;
        }
    }
    ST_PDL_WAIT();
    ST_PDL_TRIGGER();
    if (c >= channels) return;
    const int keep = taps - 1, t0 = blockIdx.x * TT;
    // N tokens from t on, all of request b; u[K - 1 + k]: the input of token t + k
    auto run = [&](auto n_const, int t, int b) {
        constexpr int N = decltype(n_const)::value;
        const int i = t - q_start[b];
        float* st = state + (size_t)slots[b] * keep * channels + c;
        ConvRaw<T, V> raw[N];
#pragma unroll
        for (int k = 0; k < N; ++k) raw[k].load(in + (size_t)(t + k) * ld + c);
        float u[K][V];                                  // the inputs of a token and the K - 1 before it
#pragma unroll
        for (int r = 0; r < K - 1; ++r) {
            const int back = K - 1 - r;                 // tokens before t
#pragma unroll
            for (int v = 0; v < V; ++v) u[r][v] = 0.f;
            if (back <= i) { if (back <= keep) load_v<V>(in + (size_t)(t - back) * ld + c, u[r]); }
            else if (back <= keep) load_v<V>(st + (size_t)(keep + i - back) * channels, u[r]);
        }
#pragma unroll
        for (int k = 0; k < N; ++k) {
            raw[k].widen(u[K - 1]);
            float y[V];
#pragma unroll
            for (int v = 0; v < V; ++v) {
                y[v] = bv[v];
#pragma unroll
                for (int j = 0; j < K; ++j) y[v] = fmaf(wv[v][j], u[j][v], y[v]);
                y[v] = apply_act(y[v], act);
            }
            store_v<V>(out + (size_t)(t + k) * channels + c, y);
            if (N == 1) break;
#pragma unroll
            for (int j = 0; j + 1 < K; ++j)
#pragma unroll
                for (int v = 0; v < V; ++v) u[j][v] = u[j + 1][v];
        }
        if (N == 1 && move_state) {
#pragma unroll
            for (int r = 1; r < K; ++r)                 // the oldest kept input stands first
                if (K - 1 - r < keep) store_v<V>(st + (size_t)(keep - K + r) * channels, u[r]);
        }
    };
    if (TT > 1 && t0 + TT <= n_tokens && positions[t0] >= 0 && positions[t0 + TT - 1] >= 0 &&
        seq_of_token[t0] == seq_of_token[t0 + TT - 1]) {
        run(std::integral_constant<int, TT>{}, t0, seq_of_token[t0]);
        return;
    }
    for (int t = t0; t < min(t0 + TT, n_tokens); ++t)
        if (positions[t] >= 0) run(std::integral_constant<int, 1>{}, t, seq_of_token[t]);      // (else: padding)
}

ST_EXPORT int st_conv_act(const void* in, int ld, const float* w, const float* bias, float* state, void* out,
                          const int* positions, const int* seq_of_token, const int* q_start, const int* slots,
                          int n_tokens, int channels, int taps, int act, int move_state, int dtype, void* stream) {
    if (n_tokens <= 0) return 0;
    if (channels <= 0 || taps < 1 || ld < channels || act < 0 || act > 5) return ST_ERR_BAD_ARG;
    if (taps > CONV_MAX_TAPS) return ST_ERR_TOO_LARGE;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = channels % 4 == 0 && ld % 4 == 0 && aligned16(in) && aligned16(out) && aligned16(state);
    const int per_block = vec ? 128 * 4 : 128;
    const int tt = n_tokens > 256 ? 8 : 1;              // few tokens: a thread each; many: the inputs are fetched once
    dim3 grid((n_tokens + tt - 1) / tt, (channels + per_block - 1) / per_block);
#define CA_LAUNCH(T, V, TT)                                                                                              \
    return st_launch_pdl("conv_act", taps <= 4 ? conv_act_kernel<T, V, TT, 4> : conv_act_kernel<T, V, TT, 8>, grid, dim3(128), 0, s, (const T*)in, ld, w, bias, state, \
                         (T*)out, positions, seq_of_token, q_start, slots, n_tokens, channels, taps, act, move_state)
#define CA_PICK(T)                                                                              \
    do {                                                                                        \
        if (vec) { if (tt == 8) CA_LAUNCH(T, 4, 8); CA_LAUNCH(T, 4, 1); }                       \
        if (tt == 8) CA_LAUNCH(T, 1, 8);                                                        \
        CA_LAUNCH(T, 1, 1);                                                                     \
    } while (0)
    if (dtype == 0) CA_PICK(float);
    if (dtype == 1) CA_PICK(bf16);
    return ST_ERR_BAD_DTYPE;
#undef CA_PICK
#undef CA_LAUNCH
}

// in: [n_tokens, channels] float (in_f32) or the storage type; out: [n_tokens, channels] storage type `dtype`
ST_EXPORT int st_conv_residual(const void* in, int in_f32, const float* w, float* state, void* out,
                               const int* positions, const int* seq_of_token, const int* q_start, const int* slots,
                               int n_tokens, int channels, int taps, int residual, int dtype, void* stream) {
    if (n_tokens <= 0) return 0;
    if (channels <= 0 || taps < 1) return ST_ERR_BAD_ARG;
    if (taps > CONV_MAX_TAPS) return ST_ERR_TOO_LARGE;
    if (dtype != 0 && dtype != 1) return ST_ERR_BAD_DTYPE;
    cudaStream_t s = (cudaStream_t)stream;
    const bool vec = channels % 4 == 0 && aligned16(in) && aligned16(out) && aligned16(state);
    const int per_block = vec ? 128 * 4 : 128;
    dim3 grid(n_tokens, (channels + per_block - 1) / per_block);
#define CONV_LAUNCH(TI, TO)                                                                                           \
    do {                                                                                                              \
        if (vec) return st_launch_pdl("conv", conv_residual_kernel<TI, TO, 4>, grid, dim3(128), 0, s, (const TI*)in, w, state, \
                                      (TO*)out, positions, seq_of_token, q_start, slots, channels, taps, residual);   \
        return st_launch_pdl("conv", conv_residual_kernel<TI, TO, 1>, grid, dim3(128), 0, s, (const TI*)in, w, state, \
                             (TO*)out, positions, seq_of_token, q_start, slots, channels, taps, residual);            \
    } while (0)
    if (dtype == 0) CONV_LAUNCH(float, float);
    else if (in_f32) CONV_LAUNCH(float, bf16);
    else CONV_LAUNCH(bf16, bf16);
#undef CONV_LAUNCH
}

// in: [rows, ld] of which the first `channels` columns are the convolution's inputs
ST_EXPORT int st_conv_state_update(const void* in, int ld, float* state, const int* positions, const int* q_start,
                                   const int* slots, int n_seqs, int channels, int taps, int dtype, void* stream) {
    if (n_seqs <= 0 || taps <= 1) return 0;
    if (channels <= 0 || ld < channels) return ST_ERR_BAD_ARG;
    if (taps > CONV_MAX_TAPS) return ST_ERR_TOO_LARGE;
    cudaStream_t s = (cudaStream_t)stream;
    dim3 grid((channels + 255) / 256, n_seqs);
    if (dtype == 0) conv_state_update_kernel<float><<<grid, 256, 0, s>>>((const float*)in, ld, state, positions, q_start, slots, channels, taps);
    else if (dtype == 1) conv_state_update_kernel<bf16><<<grid, 256, 0, s>>>((const bf16*)in, ld, state, positions, q_start, slots, channels, taps);
    else return ST_ERR_BAD_DTYPE;
    return st_launch_status();
}
