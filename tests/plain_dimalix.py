"""A plain, slow implementation of the Dimalix design in numpy float64, one function per mechanism.

It shares no code with the package: it has its own safetensors reader, reads ``config.json`` as a dict and walks
whole sequences without any cache.  Notation: T tokens, W the model width, H query heads, G key/value heads, d the
key size, e the value size; N(x; w) is an RMS norm with weight w.

  layer       x <- x + a * mixer(N(x; n1)) + b * ff(N(x; n2))                    a, b: a factor per coordinate
  attention   one projection gives a head's value and, normed with all heads together and rotated, its key; a query
              sees the keys of its own chunk
  latent      one normed latent and one rotated key part per token serve every head's keys and values, in a window
  routing     softmax scores; choice by score + correction inside the groups with the largest best choice; weights are
              the bare scores over their sum; some router outputs stand for the identity
  loop        a stretch of layers runs several times; the embedding's rows are added before every pass but the first
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
def silu(z):
    return z / (1.0 + np.exp(-z))


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def rms_norm(y, weight, eps):
    return y / np.sqrt(np.mean(y * y, axis=-1, keepdims=True) + eps) * weight


# ------------------------------------------------------------------ positions
def rotation_frequencies(rot):
    """The frequency of every pair: base^(-2i/dims), and with ``scaling`` the pairs whose wavelength exceeds
    original/low turn ``factor`` times slower, those below original/high stay, a blend lies between."""
    D = rot["dims"]
    out = [rot["base"] ** (-2.0 * i / D) for i in range(D // 2)]
    sc = rot.get("scaling")
    if sc:
        for i, f in enumerate(out):
            wave = 2.0 * math.pi / f
            if wave < sc["original"] / sc["high"]:
                continue
            if wave > sc["original"] / sc["low"]:
                out[i] = f / sc["factor"]
            else:
                share = (sc["original"] / wave - sc["low"]) / (sc["high"] - sc["low"])
                out[i] = (1.0 - share) * f / sc["factor"] + share * f
    return np.asarray(out)


def rotate_neighbours(u, positions, rot):
    """u [T, heads, d]: of the first ``dims`` dimensions, 2i turns with 2i+1."""
    if not rot or not rot["dims"]:
        return u
    D = rot["dims"]
    ang = np.asarray(positions, dtype=np.float64)[:, None] * rotation_frequencies(rot)[None, :]
    c, s = np.cos(ang)[:, None, :], np.sin(ang)[:, None, :]
    out = u.copy()
    a, b = u[..., 0:D:2], u[..., 1:D:2]
    out[..., 0:D:2] = a * c - b * s
    out[..., 1:D:2] = b * c + a * s
    return out


# ------------------------------------------------------------------ masks
def seen_window(T, size):
    """[T, T]: query i sees key j when 0 <= i - j < size (None: every key up to its own)."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i - j < size) if size else True)


def seen_chunk(T, size):
    """[T, T]: query i sees key j <= i when both lie in the same run of ``size`` positions (None: every j <= i)."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    return (j <= i) & ((i // size == j // size) if size else True)


def mask_size(mx):
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


def grouped_qkv(h, w, p, mx, eps, positions):
    """-> q [T, H, d], k [T, G, d], v [T, G, d]: the value is the key projection (bias in) itself; queries and keys are
    normed over all heads together, then rotated."""
    T = h.shape[0]
    H, G, d = mx["heads"], mx["kv_heads"], mx["dim"]
    q = h @ w[p + "q"].T + w[p + "q.b"]
    k = h @ w[p + "k"].T + w[p + "k.b"]
    v = k.reshape(T, G, d)
    q = rms_norm(q, w[p + "q.norm"], eps).reshape(T, H, d)
    k = rms_norm(k, w[p + "k.norm"], eps).reshape(T, G, d)
    return rotate_neighbours(q, positions, mx.get("rot")), rotate_neighbours(k, positions, mx.get("rot")), v


def grouped_attention(h, w, p, mx, eps):
    T = h.shape[0]
    q, k, v = grouped_qkv(h, w, p, mx, eps, np.arange(T))
    o = attend(q, k, v, seen_chunk(T, mask_size(mx)), mx["scale"])
    return o.reshape(T, -1) @ w[p + "o"].T


def latent_attention(h, w, p, mx, eps):
    T = h.shape[0]
    H, d, r, e, kr = mx["heads"], mx["dim"], mx["rot_dim"], mx["vdim"], mx["kv_rank"]
    pos = np.arange(T)
    q = (h @ w[p + "q"].T).reshape(T, H, d + r)
    down = h @ w[p + "dkv"].T
    c = rms_norm(down[:, :kr], w[p + "dkv.norm"], eps)
    k_rot = rotate_neighbours(down[:, None, kr:], pos, mx.get("rot"))[:, 0]
    k = (c @ w[p + "uk"].T).reshape(T, H, d)
    v = (c @ w[p + "uv"].T).reshape(T, H, e)
    q_rot = rotate_neighbours(q[..., d:], pos, mx.get("rot"))
    s = (np.einsum("iad,jad->aij", q[..., :d], k) + np.einsum("iar,jr->aij", q_rot, k_rot)) * mx["scale"]
    P = softmax_seen(s, seen_window(T, mask_size(mx)))
    return np.einsum("aij,jae->iae", P, v).reshape(T, H * e) @ w[p + "o"].T


# ------------------------------------------------------------------ feed-forward
def dense_ff(h, w, p):
    return gelu_tanh(h @ w[p + "up"].T) @ w[p + "down"].T


def expert(h, w, p):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def route(z, correction, router):
    """z [T, E] router logits -> (chosen [T, top], weights [T, top])."""
    s = np.exp(z - z.max(axis=-1, keepdims=True))
    s /= s.sum(axis=-1, keepdims=True)
    choice = s + correction
    T, E = s.shape
    groups = router.get("groups")
    if groups:
        n, keep = groups["count"], groups["keep"]
        of_group = choice.reshape(T, n, E // n).max(axis=-1)
        best = np.argsort(-of_group, axis=-1, kind="stable")[:, :keep]
        open_ = np.zeros((T, n), dtype=bool)
        np.put_along_axis(open_, best, True, axis=-1)
        choice = np.where(np.repeat(open_, E // n, axis=-1), choice, -np.inf)
    chosen = np.argsort(-choice, axis=-1, kind="stable")[:, :router["top"]]
    sc = np.take_along_axis(s, chosen, axis=-1)
    return chosen, sc / (sc.sum(axis=-1, keepdims=True) + 1e-20)


def experts_ff(h, w, p, mlp):
    r = mlp["router"]
    chosen, weights = route(h @ w[p + "router"].T, w[p + "correction"], r)
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        for c, wt in zip(chosen[t], weights[t]):
            out[t] += wt * (expert(h[t], w, f"{p}e{c}.") if c < r["experts"] else h[t])
    return out


def feed_forward(h, w, p, mlp):
    return dense_ff(h, w, p) if mlp["kind"] == "dense" else experts_ff(h, w, p, mlp)


# ------------------------------------------------------------------ the model
def layer(x, w, i, spec, eps):
    p = f"l{i}."
    mixer = grouped_attention if spec["type"] == "attention" else latent_attention
    y = mixer(rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", spec["mixer"], eps) * w[p + "ls1"]
    if spec.get("mlp") is not None:
        y = y + feed_forward(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp.", spec["mlp"]) * w[p + "ls2"]
    return x + y


def layer_runs(cfg):
    """[(layer, whether the embedding's rows are added first)] in running order."""
    n, loop = len(cfg["layers"]), cfg.get("loop")
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    runs = [(i, False) for i in range(a)]
    for t in range(loop["times"]):
        runs += [(i, t > 0 and i == a) for i in range(a, b)]
    return runs + [(i, False) for i in range(b, n)]


def forward(cfg, w, tokens, return_layers=False):
    """Logits [T, vocab] of a whole sequence (and the residual rows after every layer run)."""
    eps = cfg["norm"]["eps"]
    x0 = w["embed"][np.asarray(tokens)] * (cfg["embedding"]["scale"] if cfg.get("embedding") else 1.0)
    x, after = x0, []
    for i, again in layer_runs(cfg):
        x = layer(x + x0 if again else x, w, i, cfg["layers"][i], eps)
        after.append(x)
    logits = rms_norm(x, w["final.norm"], eps) @ w["head"].T
    return (logits, np.stack(after)) if return_layers else logits


def greedy(cfg, w, prompt, n_new):
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(np.argmax(forward(cfg, w, toks)[-1])))
    return toks[len(prompt):]
