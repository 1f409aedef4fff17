"""A plain, slow implementation of the Mezinex decoder: NumPy float64, one whole sequence at a time, one function
per mechanism, no cache and no batching.  It reads the raw ``config.json`` dictionary and a dictionary of arrays by
checkpoint name, and shares nothing with the engine.

Notation: T tokens, width W; a mixer's input is h [T, W]; positions are 0 .. T-1; the stream is X [S, T, W], S
copies of the residual stream.
"""

from __future__ import annotations

import json
import os

import numpy as np

from .decoder import read_safetensors


# ---- small pieces --------------------------------------------------------------------------------

def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt(np.mean(np.square(x), axis=-1, keepdims=True) + eps)


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def softplus(z):
    return np.logaddexp(0.0, z)


def silu(z):
    return z * sigmoid(z)


def gelu_tanh(z):
    return 0.5 * z * (1.0 + np.tanh(np.sqrt(2.0 / np.pi) * (z + 0.044715 * z * z * z)))


def causal_conv(x, taps, bias):
    """Per channel: out_t = bias + sum_j taps[:, j] x_(t - (J - 1) + j), zeros before the first token."""
    T, J = x.shape[0], taps.shape[1]
    padded = np.vstack([np.zeros((J - 1, x.shape[1])), x])
    return bias + sum(taps[:, j] * padded[j:j + T] for j in range(J))


def rotate_pairs(x, dims, base, positions):
    """x [T, ..., D]: channel 2i turns with channel 2i + 1 by position * base^(-2i/dims), i < dims / 2."""
    out = x.copy()
    for i in range(dims // 2):
        angle = positions * float(base) ** (-2.0 * i / dims)
        c, s = np.cos(angle), np.sin(angle)
        if x.ndim == 3:
            c, s = c[:, None], s[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i], out[..., 2 * i + 1] = u * c - v * s, v * c + u * s
    return out


# ---- the embedding and the streams -----------------------------------------------------------------

def bigram_rows(tokens, buckets, mul_prev, mul_cur):
    """The row of the pair table that every token reads; a sequence's first token reads the last row."""
    return [buckets if t == 0 else (int(tokens[t - 1]) * mul_prev + int(tokens[t]) * mul_cur) % buckets for t in range(len(tokens))]


def embed(config, w, tokens):
    x = w["embed"][np.asarray(tokens)]
    pair = (config.get("embedding") or {}).get("bigram")
    if pair:
        x = x + w["bigram"][bigram_rows(tokens, int(pair["buckets"]), int(pair["mul_prev"]), int(pair["mul_cur"]))]
    return x


def hyper_read(streams, weights):
    """What a sublayer reads: the weighted sum of the streams."""
    return np.tensordot(weights, streams, axes=(0, 0))


def hyper_write(streams, mix, out, y):
    """New stream t = sum over s of mix[s, t] (old stream s) + out[t] y."""
    return np.einsum("st,snw->tnw", mix, streams) + out[:, None, None] * y[None]


# ---- mixers ----------------------------------------------------------------------------------------

def linear_recurrence(u, r, i, lam, gain=8.0):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t, log a_t = -gain r_t softplus(lam); returns every S_t."""
    log_a = -gain * r * softplus(lam)
    state, out = np.zeros(u.shape[1]), np.zeros_like(u)
    for t in range(u.shape[0]):
        a = np.exp(log_a[t])
        state = a * state + np.sqrt(-np.expm1(2.0 * log_a[t])) * i[t] * u[t]
        out[t] = state
    return out


def rglru(h, t, m, eps):
    blocks = int(m["blocks"])
    y = gelu_tanh(h @ t["y"].T + t["y.b"])
    u = causal_conv(h @ t["x"].T + t["x.b"], t["conv"], t["conv.b"])
    parts = u.reshape(u.shape[0], blocks, -1)
    gate = lambda name: sigmoid(np.einsum("tbi,boi->tbo", parts, t[name]) + t[name + ".b"]).reshape(u.shape)
    return (linear_recurrence(u, gate("ra"), gate("ri"), t["lam"]) * y) @ t["o"].T


def state_space(x, b, c, dt, a_log, d):
    """x [T, H, V], b and c [T, G, N], dt [T, H] (after the softplus): S_t = exp(-exp(a_log) dt) S_(t-1) + dt b_t x_t^T,
    y_t = S_t^T c_t + d x_t per head, head h reading group h // (H / G)."""
    T, H, V = x.shape
    share = H // b.shape[1]
    y = np.zeros_like(x)
    for head in range(H):
        state = np.zeros((b.shape[2], V))
        for t in range(T):
            bt, ct = b[t, head // share], c[t, head // share]
            state = np.exp(-np.exp(a_log[head]) * dt[t, head]) * state + dt[t, head] * np.outer(bt, x[t, head])
            y[t, head] = state.T @ ct + d[head] * x[t, head]
    return y


def mamba2(h, t, m, eps):
    T = h.shape[0]
    H, V, N, G, parts = (int(m[k]) for k in ("heads", "vdim", "state", "groups", "norm_groups"))
    inner = H * V
    z, xbc, dt = np.split(h @ t["in"].T, [inner, 2 * inner + 2 * G * N], axis=-1)
    xbc = silu(causal_conv(xbc, t["conv"], t["conv.b"]))
    x, b, c = np.split(xbc, [inner, inner + G * N], axis=-1)
    y = state_space(x.reshape(T, H, V), b.reshape(T, G, N), c.reshape(T, G, N), softplus(dt + t["dt_bias"]), t["A_log"], t["D"])
    y = y.reshape(T, inner) * silu(z)
    y = rms_unit(y.reshape(T, parts, -1), eps).reshape(T, inner) * t["norm"]
    return y @ t["o"].T


def latent_scores(q_plain, q_rot, k_plain, k_rot, scale):
    """[T, T] scores of one head; the rotated key part is the same for every head."""
    return (q_plain @ k_plain.T + q_rot @ k_rot.T) * scale


def causal_softmax(s):
    s = np.where(np.tril(np.ones(s.shape, dtype=bool)), s, -np.inf)
    p = np.exp(s - s.max(axis=-1, keepdims=True))
    return p / p.sum(axis=-1, keepdims=True)


def latent_attention(h, t, m, eps):
    T = h.shape[0]
    H, D, R, V, C = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    pos = np.arange(T)
    dims, base = int(m["rot"]["dims"]), float(m["rot"]["base"])
    q = (rms_unit(h @ t["dq"].T, eps) * t["dq.norm"]) @ t["uq"].T
    q = q.reshape(T, H, D + R)
    down = h @ t["dkv"].T
    latent = rms_unit(down[:, :C], eps) * t["dkv.norm"]
    k_rot = rotate_pairs(down[:, C:], dims, base, pos)
    q_rot = rotate_pairs(q[..., D:], dims, base, pos)
    k_plain = (latent @ t["uk"].T).reshape(T, H, D)
    v = (latent @ t["uv"].T).reshape(T, H, V)
    out = np.zeros((T, H, V))
    for head in range(H):
        out[:, head] = causal_softmax(latent_scores(q[:, head, :D], q_rot[:, head], k_plain[:, head], k_rot, float(m["scale"]))) @ v[:, head]
    return (out.reshape(T, H * V) * sigmoid(h @ t["g"].T)) @ t["o"].T


MIXERS = {"rglru": rglru, "mamba2": mamba2, "latent_attention": latent_attention}


def gated_ffn(h, t, mlp, eps):
    return (silu(h @ t["gate"].T) * (h @ t["up"].T)) @ t["down"].T


# ---- the model -------------------------------------------------------------------------------------

def layer_order(config):
    """The layer numbers in the order they run: the looped stretch ``times`` times in a row."""
    n, loop = len(config["layers"]), config.get("loop")
    if not loop:
        return list(range(n))
    start, stop = int(loop["start"]), int(loop["stop"])
    return list(range(start)) + list(range(start, stop)) * int(loop["times"]) + list(range(stop, n))


def forward(config, tensors, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence.  ``layers_out``: a list that receives the sum of the streams after every
    layer run."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    eps = float(config["norm"]["eps"])
    x = embed(config, w, tokens)
    streams = np.stack([x] * int(config.get("streams") or 1))
    below = lambda prefix: {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}
    for i in layer_order(config):
        layer = config["layers"][i]
        sublayers = [(1, MIXERS[layer["type"]], "mix.", layer["mixer"])]
        if layer.get("mlp"):
            sublayers.append((2, gated_ffn, "mlp.", layer["mlp"]))
        for q, fn, where, sizes in sublayers:
            read = (lambda: hyper_read(streams, w[f"l{i}.hc{q}.in"])) if config.get("streams") else (lambda: streams[0])
            y = fn(rms_unit(read(), eps) * w[f"l{i}.norm{q}"], below(f"l{i}.{where}"), sizes, eps)
            if config.get("streams"):
                streams = hyper_write(streams, w[f"l{i}.hc{q}.mix"], w[f"l{i}.hc{q}.out"], y)
            else:
                streams = streams + y
        if layers_out is not None:
            layers_out.append(streams.sum(axis=0))
    x = rms_unit(streams.sum(axis=0), eps) * w["final.norm"]
    return x @ w["head"].T * float(config.get("logit_scale", 1.0))


# ---- model folders, generation ---------------------------------------------------------------------

def load_model_dir(folder, dtype=np.float64):
    """(raw config.json dictionary, tensors by name) of a model folder."""
    with open(os.path.join(folder, "config.json"), encoding="utf-8") as fh:
        config = json.load(fh)
    return config, {k: np.asarray(v, dtype=dtype) for k, v in read_safetensors(os.path.join(folder, "model.safetensors")).items()}


def forward_logits(config, w, tokens):
    return forward(config, w, tokens)


def greedy_generate(config, w, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(np.argmax(forward(config, w, ids)[-1])))
    return ids[len(prompt):]


def generation_margins(config, w, prompt, generated):
    """For every generated token: how far its plain logit lies below the largest one at its place."""
    logits = forward(config, w, list(prompt) + list(generated))
    at = len(prompt) - 1
    return [float(logits[at + i].max() - logits[at + i, t]) for i, t in enumerate(generated)]
