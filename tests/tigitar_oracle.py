"""Plain restatement of the Tigitar decoder in NumPy float64, one function per mechanism: the oracle of the CUDA path.

Slow on purpose: every sequence is walked as a whole, the recurrence token by token, attention as a full score matrix
over expanded keys with a mask, every expert on every token. Shares no code with tenzo_b200. `cfg` is the parsed
config.json, `W` maps tensor names to float64 arrays.
"""
from __future__ import annotations

import numpy as np
from sozopel_oracle import causal_conv, f32_to_bf16, bf16_to_f64, over_rms, read_safetensors, sigmoid, silu  # noqa: F401


# ---- mechanisms -------------------------------------------------------------------------------------------------------
def unit_vectors(x):
    """x / |x| over the last axis, with 1e-6 under the root."""
    return x / np.sqrt(np.sum(x * x, axis=-1, keepdims=True) + 1e-6)


def head_decay(z, a_log, dt_bias):
    """z [T, H]: exp(-exp(a_log) * ln(1 + e^(z + dt_bias)))."""
    return np.exp(-np.exp(a_log) * np.logaddexp(0.0, z + dt_bias))


def delta_recurrence(q, k, v, decay, beta):
    """q, k [T, H, dim], v [T, H, vdim], decay, beta [T, H]. The state is decayed, corrected towards v along k, then read."""
    T, H, dim = q.shape
    S = np.zeros((H, dim, v.shape[2]))
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        S = S * decay[t][:, None, None]
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out


def rotate_halves(x, positions, base):
    """x [T, ..., dims]: element i turns with element i + dims/2 by position * base^(-2i/dims)."""
    half = x.shape[-1] // 2
    angle = np.asarray(positions, np.float64)[:, None] * base ** (-np.arange(half) / half)
    angle = angle.reshape((len(x),) + (1,) * (x.ndim - 2) + (half,))
    u, v = x[..., :half], x[..., half:]
    return np.concatenate([u * np.cos(angle) - v * np.sin(angle), v * np.cos(angle) + u * np.sin(angle)], axis=-1)


def window_softmax(scores, window):
    """scores [T, T] of queries against keys: softmax over the last `window` places, oneself included."""
    T = len(scores)
    dist = np.arange(T)[:, None] - np.arange(T)[None, :]
    s = np.where((dist >= 0) & (dist < window), scores, -np.inf)
    e = np.exp(s - s.max(axis=1, keepdims=True))
    return e / e.sum(axis=1, keepdims=True)


def latent_attention(q, rot_q, c, rot_k, uk, uv, scale, window):
    """q [T, H, dim], rot_q [T, H, rot], c [T, rank], rot_k [T, rot], uk [H, dim, rank], uv [H, vdim, rank] -> [T, H, vdim]."""
    T, H, _ = q.shape
    out = np.zeros((T, H, uv.shape[1]))
    for h in range(H):
        s = (q[:, h] @ (c @ uk[h].T).T + rot_q[:, h] @ rot_k.T) * scale
        out[:, h] = window_softmax(s, window) @ (c @ uv[h].T)
    return out


def route(z, correction, top):
    """z [T, E] -> (chosen [T, top], weights [T, top]): largest score plus correction, weighted by the score alone."""
    s = sigmoid(z)
    chosen = np.argsort(-(s + correction), axis=1, kind="stable")[:, :top]
    return chosen, np.take_along_axis(s, chosen, axis=1)


def glu(h, gate, up, down, act):
    return (act(h @ gate.T) * (h @ up.T)) @ down.T


def relu(z):
    return np.maximum(z, 0.0)


def soft_cap(z, cap):
    return cap * np.tanh(z / cap)


# ---- sublayers: h [T, width] -> [T, width] -------------------------------------------------------------------------------
def _heads(x, n):
    return x.reshape(len(x), n, -1)


def mixer_delta(h, mix, W, pre, eps):
    n, kv = mix["heads"], mix["kv_heads"]
    q, k, v = (silu(causal_conv(h @ W[pre + s].T, W[pre + s + ".conv"])) for s in "qkv")
    q, k = (np.repeat(unit_vectors(_heads(x, kv)), n // kv, axis=1) for x in (q, k))
    decay = head_decay(h @ W[pre + "a"].T, W[pre + "A_log"], W[pre + "dt_bias"])
    o = delta_recurrence(q * mix["dim"] ** -0.5, k, _heads(v, n), decay, sigmoid(h @ W[pre + "b"].T))
    o = over_rms(o, eps) * W[pre + "norm"]
    return (o.reshape(len(h), -1) * silu(h @ W[pre + "g"].T)) @ W[pre + "o"].T


def latent_of(h, mix, W, pre, eps):
    """The latent and the rotated key part of every token."""
    rank = mix["kv_rank"]
    y = h @ W[pre + "dkv"].T
    return over_rms(y[:, :rank], eps) * W[pre + "dkv.norm"], rotate_halves(y[:, rank:], range(len(h)), mix["rot"]["base"])


def mixer_latent(h, mix, W, pre, latent):
    n, dim = mix["heads"], mix["dim"]
    q = _heads(h @ W[pre + "q"].T, n)
    rot_q = rotate_halves(q[:, :, dim:], range(len(h)), mix["rot"]["base"])
    o = latent_attention(q[:, :, :dim], rot_q, *latent, _heads(W[pre + "uk"].T, n).transpose(1, 2, 0),
                         _heads(W[pre + "uv"].T, n).transpose(1, 2, 0), mix["scale"], mix["mask"]["size"])
    return o.reshape(len(h), -1) @ W[pre + "o"].T


def feed_forward(h, mlp, W, pre):
    if mlp["kind"] == "dense":
        return glu(h, W[pre + "gate"], W[pre + "up"], W[pre + "down"], relu)
    chosen, weights = route(h @ W[pre + "router"].T, W[pre + "correction"], mlp["router"]["top"])
    y = np.zeros_like(h)
    for e in range(mlp["router"]["experts"]):
        share = np.where(chosen == e, weights, 0.0).sum(axis=1, keepdims=True)
        y += share * glu(h, *(W[f"{pre}e{e}.{s}"] for s in ("gate", "up", "down")), silu)
    return y


# ---- the model --------------------------------------------------------------------------------------------------------
def forward(cfg, W, tokens, layers_out=None):
    """Logits [T, vocab] of one whole sequence; layers_out collects the residual after every layer."""
    eps = cfg["norm"]["eps"]
    norm = lambda x, name: over_rms(x, eps) * W[name]
    x = W["embed"][np.asarray(tokens)]
    latents = {}
    for i, layer in enumerate(cfg["layers"]):
        p, mix = f"l{i}.", layer["mixer"]
        h = norm(x, p + "norm1")
        if layer["type"] == "delta":
            y = mixer_delta(h, mix, W, p + "mix.", eps)
        else:
            if "kv_from" not in mix:
                latents[i] = latent_of(h, mix, W, p + "mix.", eps)
            y = mixer_latent(h, mix, W, p + "mix.", latents[mix.get("kv_from", i)])
        x = x + norm(y, p + "norm1b")
        if layer["mlp"] is not None:
            x = x + norm(feed_forward(norm(x, p + "norm2"), layer["mlp"], W, p + "mlp."), p + "norm2b")
        if layers_out is not None:
            layers_out.append(x.copy())
    return soft_cap(norm(x, "final.norm") @ W["head"].T, cfg["logit_softcap"])


def greedy(cfg, W, prompt, n):
    seq = [int(t) for t in prompt]
    for _ in range(n):
        seq.append(int(np.argmax(forward(cfg, W, seq)[-1])))
    return seq[len(prompt):]
