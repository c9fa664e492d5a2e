"""Plain restatement of the Sozopel decoder in NumPy float64, one function per mechanism: the oracle of the CUDA path.

Slow on purpose: every sequence is walked as a whole, recurrences token by token, attention as a full score matrix with a
mask. Shares no code with tenzo_b200. `cfg` is the parsed config.json, `W` maps tensor names to float64 arrays.
"""
from __future__ import annotations

import json
import struct
from pathlib import Path

import numpy as np


# ---- files ------------------------------------------------------------------------------------------------------------
def bf16_to_f64(raw: np.ndarray) -> np.ndarray:
    return (raw.astype(np.uint32) << 16).view(np.float32).astype(np.float64)


def f32_to_bf16(x: np.ndarray) -> np.ndarray:
    """Round to nearest even; returns the 16-bit patterns."""
    b = np.ascontiguousarray(x, np.float32).view(np.uint32)
    return ((b + 0x7FFF + ((b >> 16) & 1)) >> 16).astype(np.uint16)


def read_safetensors(path) -> dict:
    data = Path(path).read_bytes()
    n = struct.unpack("<Q", data[:8])[0]
    out = {}
    for name, e in json.loads(data[8:8 + n]).items():
        if name == "__metadata__":
            continue
        a, b = e["data_offsets"]
        buf = data[8 + n + a:8 + n + b]
        arr = bf16_to_f64(np.frombuffer(buf, np.uint16)) if e["dtype"] == "BF16" else np.frombuffer(buf, np.int32).astype(np.float64)
        out[name] = arr.reshape(e["shape"])
    return out


# ---- mechanisms -------------------------------------------------------------------------------------------------------
def over_rms(x, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return np.exp(-np.logaddexp(0.0, -z))


def silu(z):
    return z * sigmoid(z)


def causal_conv(u, w):
    """u [T, C], w [C, taps]: tap j multiplies the input taps - 1 - j steps back; missing inputs count as 0."""
    taps = w.shape[1]
    padded = np.concatenate([np.zeros((taps - 1, u.shape[1])), u])
    return sum(w[:, j] * padded[j:j + len(u)] for j in range(taps))


def xielu(z, p, q):
    pos, neg = np.logaddexp(0.0, p), 0.5 + np.logaddexp(0.0, q)
    return np.where(z > 0, pos * z * z, neg * (np.expm1(np.minimum(z, 0.0)) - z)) + 0.5 * z


def window_attention(q, k, v, scale, window):
    """q [T, H, dim], k [T, G, dim], v [T, G, vdim]: distance bias, window, unit sink in the softmax."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = np.zeros((T, H, v.shape[2]))
    dist = np.arange(T)[:, None] - np.arange(T)[None, :]
    seen = (dist >= 0) & (dist < window)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale - 2.0 ** (-8.0 * (h + 1) / H) * dist
        s = np.where(seen, s, -np.inf)
        m = np.maximum(s.max(axis=1, keepdims=True), 0.0)
        e = np.exp(s - m)
        out[:, h] = (e @ v[:, g]) / (np.exp(-m) + e.sum(axis=1, keepdims=True))
    return out


def linear_recurrence(q, k, v, decay, bonus=None):
    """q, k, decay [T, H, dim], v [T, H, vdim]. Without bonus the output reads the state after the update, with it the
    state before the update plus diag(bonus) k v^T."""
    T, H, dim = q.shape
    S = np.zeros((H, dim, v.shape[2]))
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        kv = k[t][:, :, None] * v[t][:, None, :]
        new = decay[t][:, :, None] * S + kv
        read = new if bonus is None else S + bonus[:, :, None] * kv
        out[t] = np.einsum("hd,hdv->hv", q[t], read)
        S = new
    return out


# ---- mixers: h [T, width] -> [T, width] ---------------------------------------------------------------------------------
def _heads(x, n):
    return x.reshape(len(x), n, -1)


def mixer_retention(h, mix, W, pre, eps):
    n = mix["heads"]
    q, k, v = (_heads(h @ W[pre + s].T, n) for s in ("q", "k", "v"))
    k = k * mix["dim"] ** -0.5
    decay = np.broadcast_to(np.asarray(mix["decay"], np.float64)[None, :, None], k.shape)
    o = over_rms(linear_recurrence(q, k, v, decay), eps)
    return (o.reshape(len(h), -1) * silu(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def mixer_wkv(h, mix, W, pre, eps):
    n = mix["heads"]
    prev = np.concatenate([np.zeros((1, h.shape[1])), h[:-1]])
    m = {s: h + (prev - h) * W[pre + "mu." + s] for s in "rkvgw"}
    r, k, v = (_heads(m[s] @ W[pre + s].T, n) for s in "rkv")
    z = np.tanh(m["w"] @ W[pre + "w1"].T) @ W[pre + "w2"].T + W[pre + "w0"]
    decay = _heads(np.exp(-np.exp(z)), n)
    o = over_rms(linear_recurrence(r, k, v, decay, bonus=W[pre + "u"].reshape(n, -1)), eps)
    return (o.reshape(len(h), -1) * W[pre + "norm"] * silu(m["g"] @ W[pre + "g"].T)) @ W[pre + "o"].T


def parallel_left(h, mix, W, pre):
    H, G = mix["heads"], mix["kv_heads"]
    q, k, v = (causal_conv(h @ W[pre + s].T, W[pre + s + ".conv"]) for s in ("q", "k", "v"))
    o = window_attention(_heads(q, H), _heads(k, G), _heads(v, G), mix["scale"], mix["mask"]["size"])
    return o.reshape(len(h), -1) @ W[pre + "o"].T


def parallel_right(h, mix, W, pre, eps):
    n = mix["heads"]
    q, k, v = (_heads(h @ W[pre + s].T, n) for s in ("q", "k", "v"))
    z = (h @ W[pre + "a1"].T) @ W[pre + "a2"].T + W[pre + "a2.b"]
    alpha = _heads(np.exp(-np.logaddexp(0.0, -z) / mix["tau"]), n)
    o = over_rms(linear_recurrence(q * mix["dim"] ** -0.5, k, v, alpha), eps) * W[pre + "norm"]
    return (o.reshape(len(h), -1) * silu(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def mixer_parallel(h, mix, W, pre, eps):
    left = over_rms(parallel_left(h, mix["left"], W, pre + "left."), eps) * W[pre + "left.out"]
    right = over_rms(parallel_right(h, mix["right"], W, pre + "right.", eps), eps) * W[pre + "right.out"]
    return 0.5 * (left + right)


MIXERS = {"retention": mixer_retention, "wkv": mixer_wkv, "parallel": mixer_parallel}


def dense_ff(h, W, pre):
    return xielu(h @ W[pre + "up"].T, *W[pre + "act"]) @ W[pre + "down"].T


# ---- the model --------------------------------------------------------------------------------------------------------
def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence; layers_out collects the residual after every layer."""
    eps = cfg["norm"]["eps"]
    tokens = np.asarray(tokens)
    x = W["embed"][tokens] + W["pos"][:len(tokens)]

    def sublayer_input(x, norm, conv):
        h = over_rms(x, eps) * W[norm]
        return h + causal_conv(h, W[conv])

    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[layer["type"]](sublayer_input(x, p + "norm1", p + "canon1"), layer["mixer"], W, p + "mix.", eps)
        if layer["mlp"] is not None:
            x = x + dense_ff(sublayer_input(x, p + "norm2", p + "canon2"), W, p + "mlp.")
        if layers_out is not None:
            layers_out.append(x.copy())
    return (over_rms(x, eps) * W["final.norm"]) @ W["head"].T


def greedy(cfg, W, prompt, n):
    seq = [int(t) for t in prompt]
    for _ in range(n):
        seq.append(int(np.argmax(forward(cfg, W, seq)[-1])))
    return seq[len(prompt):]
