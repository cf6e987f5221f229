"""A plain, slow implementation of the Nigilorn design in numpy float64, one function per mechanism.

It shares no code with the package: it has its own safetensors reader, reads ``config.json`` as a dict and walks
whole sequences without any cache.  Notation: T tokens, W the model width, H query heads, G key/value heads, d the
key size, e the value size, C inner channels, N state size; N(x; w) is an RMS norm with weight w.

  sub-layer   h = N(x; n);  x <- x + N( sigmoid(R h + r) * f(h); n' )            f: the mixer, then the feed-forward
  side input  x <- x + N( P (gelu_tanh(K x) * e_token); s )                      e_token: the layer's part of a table row
  scan        S[c, n] <- exp(-t_c exp(a[c, n])) S[c, n] + t_c u_c b_n;  y_c = sum_n S[c, n] g_n + D_c u_c
  latent      one normed latent and one rotated key part per token serve every head's keys and values
  routing     sigmoid scores; the best groups by the sum of their two largest; the largest scores inside those
"""
from __future__ import annotations

import json
import math
import os
import struct

import numpy as np


def read_safetensors(path):
    with open(path, "rb") as f:
        (n,) = struct.unpack("<Q", f.read(8))
        meta = json.loads(f.read(n))
        data = f.read()
    out = {}
    for name, info in meta.items():
        if name == "__metadata__":
            continue
        lo, hi = info["data_offsets"]
        raw, shape = data[lo:hi], info["shape"]
        if info["dtype"] == "BF16":
            a = (np.frombuffer(raw, dtype="<u2").astype(np.uint32) << 16).view(np.float32).astype(np.float64)
        elif info["dtype"] == "F32":
            a = np.frombuffer(raw, dtype="<f4").astype(np.float64)
        elif info["dtype"] == "I32":
            a = np.frombuffer(raw, dtype="<i4").astype(np.int64)
        else:
            raise ValueError(f"{name}: unexpected dtype {info['dtype']}")
        out[name] = a.reshape(shape)
    return out


def load_model(model_dir):
    with open(os.path.join(model_dir, "config.json")) as f:
        cfg = json.load(f)
    return cfg, read_safetensors(os.path.join(model_dir, "model.safetensors"))


# ------------------------------------------------------------------ elementary functions
def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return np.logaddexp(0.0, z)


def relu2(z):
    return np.maximum(z, 0.0) ** 2


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_unit(y, eps):
    """y divided by its root mean square over the last axis, eps inside the root."""
    return y / np.sqrt(np.mean(y * y, axis=-1, keepdims=True) + eps)


def causal_conv(u, f, b):
    """out_t = b + sum_j f[:, j] u_(t - taps + 1 + j), zeros before the start.  u [T, C], f [C, taps], b [C]."""
    T, taps = u.shape[0], f.shape[1]
    out = np.repeat(b[None], T, axis=0).astype(np.float64)
    for j in range(taps):
        back = taps - 1 - j
        if back < T:
            out[back:] += f[:, j] * u[:T - back]
    return out


# ------------------------------------------------------------------ positions
def rotation_frequencies(rot):
    """(frequency of every pair, amplitude of the sines): base^(-2i/dims), slowed down by ``factor`` for the pairs
    that turn rarely within the original context, with a linear ramp between the two regimes."""
    D, base = rot["dims"], rot["base"]
    i = np.arange(D // 2, dtype=np.float64)
    freq = base ** (-2.0 * i / D)
    sc = rot.get("scaling")
    if not sc:
        return freq, 1.0
    pair_with_turns = lambda t: D * math.log(sc["original"] / (2 * math.pi * t)) / (2 * math.log(base))
    first = max(math.floor(pair_with_turns(sc["fast"])), 0)
    last = min(math.ceil(pair_with_turns(sc["slow"])), D - 1)
    ramp = np.clip((i - first) / max(last - first, 0.001), 0.0, 1.0)
    return freq / sc["factor"] * ramp + freq * (1.0 - ramp), 0.1 * math.log(sc["factor"]) + 1.0


def rotate_neighbours(u, positions, rot):
    """u [T, heads, d]: of the first ``dims`` dimensions, 2i turns with 2i+1."""
    if not rot or not rot["dims"]:
        return u
    D = rot["dims"]
    freq, amp = rotation_frequencies(rot)
    ang = np.asarray(positions, dtype=np.float64)[:, None] * freq[None, :]
    c, s = amp * np.cos(ang)[:, None, :], amp * np.sin(ang)[:, None, :]
    out = u.copy()
    a, b = u[..., 0:D:2], u[..., 1:D:2]
    out[..., 0:D:2] = a * c - b * s
    out[..., 1:D:2] = b * c + a * s
    return out


def seen_window(T, size):
    """[T, T]: query i sees key j when 0 <= i - j < size (size None: every earlier key and itself)."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (i - j >= 0) & ((i - j < size) if size else True)


def window_of(mx):
    return mx["mask"]["size"] if mx.get("mask") else None


def softmax_seen(s, seen):
    s = np.where(seen[None], s, -np.inf)
    p = np.exp(s - s.max(axis=-1, keepdims=True))
    return p / p.sum(axis=-1, keepdims=True)


# ------------------------------------------------------------------ mixers
def attend(q, k, v, seen, scale):
    """q [T, H, d], k [T, G, d], v [T, G, e] -> [T, H, e]; head a reads group a // (H / G)."""
    H, G = q.shape[1], k.shape[1]
    grp = np.arange(H) // (H // G)
    P = softmax_seen(np.einsum("iad,jad->aij", q, k[:, grp, :]) * scale, seen)
    return np.einsum("aij,jae->iae", P, v[:, grp, :])


def gated_attention(h, w, p, mx, eps):
    T = h.shape[0]
    H, G, d, e = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"]
    pos = np.arange(T)
    q = rms_unit(rotate_neighbours((h @ w[p + "q"].T).reshape(T, H, d), pos, mx.get("rot")), eps)
    k = rms_unit(rotate_neighbours((h @ w[p + "k"].T).reshape(T, G, d), pos, mx.get("rot")), eps)
    v = (h @ w[p + "v"].T).reshape(T, G, e)
    o = attend(q, k, v, seen_window(T, window_of(mx)), mx["scale"])
    o = o * sigmoid(h @ w[p + "g"].T)[:, :, None]
    return o.reshape(T, H * e) @ w[p + "o"].T


def latent_attention(h, w, p, mx, eps):
    T = h.shape[0]
    H, d, r, e, kr = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    pos = np.arange(T)
    q = (h @ w[p + "q"].T).reshape(T, H, d + r)
    down = h @ w[p + "dkv"].T
    c = rms_unit(down[:, :kr], eps) * w[p + "dkv.norm"]
    k_rot = rotate_neighbours(down[:, None, kr:], pos, mx.get("rot"))[:, 0]
    k = (c @ w[p + "uk"].T).reshape(T, H, d)
    v = (c @ w[p + "uv"].T).reshape(T, H, e)
    q_rot = rotate_neighbours(q[..., d:], pos, mx.get("rot"))
    s = (np.einsum("iad,jad->aij", q[..., :d], k) + np.einsum("iar,jr->aij", q_rot, k_rot)) * mx["scale"]
    P = softmax_seen(s, seen_window(T, window_of(mx)))
    return np.einsum("aij,jae->iae", P, v).reshape(T, H * e) @ w[p + "o"].T


def selective_scan(u, dt, a_log, b, g, D, S=None):
    """u, dt [T, C]; a_log [C, N]; b, g [T, N]; D [C] -> (y [T, C], the last state [C, N])."""
    T, C = u.shape
    S = np.zeros(a_log.shape) if S is None else S.copy()
    A = -np.exp(a_log)
    y = np.zeros((T, C))
    for t in range(T):
        S = np.exp(dt[t][:, None] * A) * S + (dt[t] * u[t])[:, None] * b[t][None, :]
        y[t] = S @ g[t] + D * u[t]
    return y, S


def mamba(h, w, p, mx):
    C, N, R = mx["inner"], mx["state"], mx["dt_rank"]
    both = h @ w[p + "in"].T
    u, z = silu(causal_conv(both[:, :C], w[p + "conv"], w[p + "conv.b"])), both[:, C:]
    xd = u @ w[p + "x"].T
    dt = softplus(xd[:, :R] @ w[p + "dt"].T + w[p + "dt.b"])
    y, _ = selective_scan(u, dt, w[p + "A_log"], xd[:, R:R + N], xd[:, R + N:], w[p + "D"])
    return (y * silu(z)) @ w[p + "o"].T


# ------------------------------------------------------------------ feed-forward
def dense_ff(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def relu2_ff(h, w, p):
    return relu2(h @ w[p + "up"].T) @ w[p + "down"].T


def route(h, w_router, router):
    """-> (chosen [T, top], weights [T, top])."""
    s = sigmoid(h @ w_router.T)
    T, E = s.shape
    top, groups = router["top"], router.get("groups")
    allowed = np.ones((T, E), dtype=bool)
    if groups:
        n = groups["count"]
        by_group = np.sort(s.reshape(T, n, E // n), axis=-1)[..., ::-1]
        score = by_group[..., :2].sum(-1)
        best = np.argsort(-score, axis=-1, kind="stable")[:, :groups["keep"]]
        keep = np.zeros((T, n), dtype=bool)
        np.put_along_axis(keep, best, True, axis=-1)
        allowed = np.repeat(keep, E // n, axis=-1)
    chosen = np.argsort(-np.where(allowed, s, -1.0), axis=-1, kind="stable")[:, :top]
    sc = np.take_along_axis(s, chosen, axis=-1)
    return chosen, sc / (sc.sum(-1, keepdims=True) + 1e-20) * router.get("scale", 1.0)


def experts_ff(h, w, p, mlp):
    chosen, weights = route(h, w[p + "router"], mlp["router"])
    out = relu2_ff(h, w, p + "shared.") if mlp.get("shared") else np.zeros_like(h)
    for t in range(h.shape[0]):
        for c, wt in zip(chosen[t], weights[t]):
            out[t] += wt * relu2_ff(h[t], w, f"{p}e{c}.")
    return out


def feed_forward(h, w, p, mlp):
    return dense_ff(h, w, p) if mlp["kind"] == "dense" else experts_ff(h, w, p, mlp)


# ------------------------------------------------------------------ the model
def mixer(h, w, p, layer, eps):
    mx = layer["mixer"]
    if layer["type"] == "mamba1":
        return mamba(h, w, p, mx)
    return (gated_attention if layer["type"] == "attention" else latent_attention)(h, w, p, mx, eps)


def sublayer(x, f, w, norm_in, gate, norm_out, eps):
    """x + N(sigmoid(R h + r) * f(h)) with h = N(x)."""
    h = rms_unit(x, eps) * w[norm_in]
    return x + rms_unit(sigmoid(h @ w[gate].T + w[gate + ".b"]) * f(h), eps) * w[norm_out]


def side_input(x, w, p, e, eps):
    y = (gelu_tanh(x @ w[p + "gate"].T) * e) @ w[p + "proj"].T
    return x + rms_unit(y, eps) * w[p + "norm"]


def forward(cfg, w, tokens, return_layers=False):
    """Logits [T, vocab] of a whole sequence (and the residual rows after every layer)."""
    eps = cfg["norm"]["eps"]
    tokens = np.asarray(tokens)
    x = w["embed"][tokens]
    after = []
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = sublayer(x, lambda h: mixer(h, w, p + "mix.", layer, eps), w, p + "norm1", p + "rg1", p + "norm1b", eps)
        if layer.get("mlp") is not None:
            x = sublayer(x, lambda h: feed_forward(h, w, p + "mlp.", layer["mlp"]), w, p + "norm2", p + "rg2",
                         p + "norm2b", eps)
        if cfg.get("token_side"):
            n = cfg["token_side"]["dim"]
            x = side_input(x, w, p + "side.", w["side.embed"][tokens][:, i * n:(i + 1) * n], eps)
        after.append(x)
    logits = (rms_unit(x, eps) * w["final.norm"]) @ w["head"].T
    return (logits, np.stack(after)) if return_layers else logits


def greedy(cfg, w, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(np.argmax(forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]
