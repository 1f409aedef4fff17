"""A plain, slow implementation of the Sudilorn decoder: NumPy float64, one whole sequence at a time, one function
per mechanism, no cache and no batching.  It reads the raw ``config.json`` dictionary and a dictionary of arrays by
checkpoint name, and shares nothing with the engine.

Notation: T tokens, width W; the stream is x [T, W]; a mixer's input is h [T, W]; positions are 0 .. T-1.
"""

from __future__ import annotations

import json
import math
import os

import numpy as np

from .decoder import read_safetensors


# ---- small pieces --------------------------------------------------------------------------------

def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / np.sqrt(np.mean(np.square(x), axis=-1, keepdims=True) + eps)


def centred_norm(x, w, eps):
    """RMS norm whose weight is kept as its distance from one."""
    return rms_unit(x, eps) * (1.0 + w)


def sigmoid(z):
    return np.where(z >= 0, 1.0 / (1.0 + np.exp(-np.abs(z))), np.exp(-np.abs(z)) / (1.0 + np.exp(-np.abs(z))))


def softplus(z):
    return np.logaddexp(0.0, z)


def silu(z):
    return z * sigmoid(z)


def causal_conv(x, taps):
    """Per channel: out_t = sum_j taps[:, j] x_(t - (J - 1) + j), zeros before the first token."""
    T, J = x.shape[0], taps.shape[1]
    padded = np.vstack([np.zeros((J - 1, x.shape[1])), x])
    return sum(taps[:, j] * padded[j:j + T] for j in range(J))


# ---- rotation ---------------------------------------------------------------------------------------

def ramp_frequencies(dims, base, scaling):
    """(frequencies [dims / 2], magnitude); ``scaling`` None or a dict with factor, original, fast, slow."""
    f = np.array([float(base) ** (-2.0 * i / dims) for i in range(dims // 2)])
    if not scaling:
        return f, 1.0
    factor, original = float(scaling["factor"]), float(scaling["original"])
    turns = lambda t: dims * math.log(original / (2.0 * math.pi * float(t))) / (2.0 * math.log(float(base)))
    lo, hi = max(math.floor(turns(scaling["fast"])), 0), min(math.ceil(turns(scaling["slow"])), dims - 1)
    ramp = np.clip((np.arange(dims // 2) - lo) / max(hi - lo, 0.001), 0.0, 1.0)
    return f / factor * ramp + f * (1.0 - ramp), 0.1 * math.log(factor) + 1.0


def rotate(x, rot, layout):
    """x [T, heads, D]: the first rot.dims channels of every head turn with the token's position; ``layout`` "halves"
    pairs channel i with i + dims / 2, "pairs" channel 2i with 2i + 1."""
    dims = int((rot or {}).get("dims") or 0)
    if not dims:
        return x
    f, mag = ramp_frequencies(dims, rot["base"], rot.get("scaling"))
    out, pos = x.copy(), np.arange(x.shape[0])
    for i in range(dims // 2):
        a, b = (i, i + dims // 2) if layout == "halves" else (2 * i, 2 * i + 1)
        c, s = mag * np.cos(pos * f[i])[:, None], mag * np.sin(pos * f[i])[:, None]
        u, v = x[..., a], x[..., b]
        out[..., a], out[..., b] = u * c - v * s, v * c + u * s
    return out


# ---- softmax attention -------------------------------------------------------------------------------

def visible(T, mask):
    """[T, T]: which keys (columns) every query sees; ``mask`` None, or a window ``size`` beside ``keep_first`` tokens."""
    i, j = np.arange(T)[:, None], np.arange(T)[None, :]
    ok = j <= i
    size = int((mask or {}).get("size") or 0)
    return ok & ((i - j < size) | (j < int(mask.get("keep_first") or 0))) if size else ok


def softmax_attention(q, k, v, scale, seen):
    """One head: q [T, D], k [T, D], v [T, V]."""
    s = np.where(seen, (q @ k.T) * scale, -np.inf)
    p = np.exp(s - s.max(axis=-1, keepdims=True))
    return (p / p.sum(axis=-1, keepdims=True)) @ v


def mixing_weight(t, diff):
    """The weight of a differential attention's second map."""
    return math.exp(float(np.sum(t["lq1"] * t["lk1"]))) - math.exp(float(np.sum(t["lq2"] * t["lk2"]))) + float(diff)


def differential_heads(a1, a2, lam, diff, eps):
    """a1, a2 [..., V]: the heads' results on the two maps."""
    return rms_unit(a1 - lam * a2, eps) * (1.0 - float(diff))


def differential_attention(h, t, m, eps):
    T, H, D = h.shape[0], int(m["heads"]), int(m["dim"])
    G, V = int(m.get("kv_heads") or H), int(m.get("vdim") or D)
    proj = {n: h @ t[n].T for n in "qkv"}
    if m.get("conv"):
        proj = {n: causal_conv(proj[n], t[n + ".conv"]) for n in proj}
    unit = lambda x, name: rotate(rms_unit(x.reshape(T, -1, D), eps) * t[name], m.get("rot"), "halves")
    q, k = unit(proj["q"], "q.norm").reshape(T, H, 2, D), unit(proj["k"], "k.norm").reshape(T, G, 2, D)
    v, seen = proj["v"].reshape(T, G, V), visible(T, m.get("mask"))
    maps = np.zeros((2, T, H, V))
    for a in range(2):
        for head in range(H):
            g = head // (H // G)
            maps[a, :, head] = softmax_attention(q[:, head, a], k[:, g, a], v[:, g], float(m["scale"]), seen)
    o = differential_heads(maps[0], maps[1], mixing_weight(t, m["diff"]), m["diff"], eps)
    return (o.reshape(T, H * V) * sigmoid(h @ t["g"].T)) @ t["o"].T


def window_attention(h, t, m, eps):
    T, H, D = h.shape[0], int(m["heads"]), int(m["dim"])
    G, V = int(m.get("kv_heads") or H), int(m.get("vdim") or D)
    turn = lambda n: rotate((h @ t[n].T + t[n + ".b"]).reshape(T, -1, D), m.get("rot"), "pairs")
    q, k, v = turn("q"), turn("k"), (h @ t["v"].T + t["v.b"]).reshape(T, G, V)
    seen = visible(T, m.get("mask"))
    out = np.stack([softmax_attention(q[:, i], k[:, i // (H // G)], v[:, i // (H // G)], float(m["scale"]), seen) for i in range(H)], axis=1)
    return out.reshape(T, H * V) @ t["o"].T


# ---- the gated delta rule ------------------------------------------------------------------------------

def delta_rule(q, k, v, beta, decay, state=None):
    """q, k [T, H, D], v [T, H, V], beta, decay [T, H]: S <- decay S, then a write of beta (v - S^T k) along k, then
    the read-out S^T q; returns what is read, [T, H, V], and the state after the last token."""
    T, H, V = v.shape
    S = np.zeros((H, k.shape[2], V)) if state is None else state.copy()
    out = np.zeros_like(v)
    for t in range(T):
        S *= decay[t][:, None, None]
        u = beta[t][:, None] * (v[t] - np.einsum("hdv,hd->hv", S, k[t]))
        S += k[t][:, :, None] * u[:, None, :]
        out[t] = np.einsum("hdv,hd->hv", S, q[t])
    return out, S


def unit_vectors(x):
    return x / np.sqrt(np.sum(np.square(x), axis=-1, keepdims=True) + 1e-6)


def gated_delta(h, t, m, eps):
    T, H, D, V = h.shape[0], int(m["heads"]), int(m["dim"]), int(m["vdim"])
    G = int(m.get("kv_heads") or H)
    short = lambda n: silu(causal_conv(h @ t[n].T, t[n + ".conv"]))
    of_head = np.arange(H) // (H // G)
    q = unit_vectors(short("q").reshape(T, G, D))[:, of_head] * D ** -0.5
    k = unit_vectors(short("k").reshape(T, G, D))[:, of_head]
    beta = sigmoid(h @ t["b"].T)
    decay = np.exp(-np.exp(t["A_log"]) * softplus(h @ t["a"].T + t["dt_bias"]))
    o, _ = delta_rule(q, k, short("v").reshape(T, H, V), beta, decay)
    o = rms_unit(o, eps) * t["norm"] * silu((h @ t["g"].T).reshape(T, H, V))
    return o.reshape(T, H * V) @ t["o"].T


def parallel_mixer(h, t, m, eps):
    below = lambda p: {k[len(p):]: v for k, v in t.items() if k.startswith(p)}
    return (float(m.get("left_scale", 1.0)) * window_attention(h, below("left."), m["left"], eps)
            + float(m.get("right_scale", 1.0)) * gated_delta(h, below("right."), m["right"], eps))


MIXERS = {"attention": differential_attention, "parallel": parallel_mixer}


# ---- the routed feed-forward ------------------------------------------------------------------------------

def relu2_expert(h, up, down):
    return np.square(np.maximum(h @ up.T, 0.0)) @ down.T


def route(z, correction, r):
    """z [E]: one token's router logits.  Returns (the chosen experts, their weights)."""
    E, top = int(r["experts"]), int(r["top"])
    groups = r.get("groups") or {}
    count = int(groups.get("count") or 1)
    keep = int(groups.get("keep") or count)
    s = sigmoid(z)
    choice = s + correction
    marks = np.array([np.sort(part)[::-1][:2].sum() for part in choice.reshape(count, E // count)])
    kept = np.argsort(-marks, kind="stable")[:keep]
    choice = np.where(np.isin(np.arange(E) // (E // count), kept), choice, -np.inf)
    chosen = np.argsort(-choice, kind="stable")[:top]
    return chosen, s[chosen]


def routed_ffn(h, t, mlp):
    out = np.zeros_like(h)
    z = h @ t["router"].T
    for n in range(h.shape[0]):
        for e, w in zip(*route(z[n], t["correction"], mlp["router"])):
            out[n] += w * relu2_expert(h[n], t[f"e{e}.up"], t[f"e{e}.down"])
    return out


# ---- the model -------------------------------------------------------------------------------------

def forward(config, tensors, tokens, layers_out=None):
    """Logits [T, vocab] of one sequence.  ``layers_out``: a list that receives the stream after every layer."""
    w = {k: np.asarray(v, dtype=np.float64) for k, v in tensors.items()}
    eps, m = float(config["norm"]["eps"]), float(config.get("residual_mult", 1.0))
    below = lambda p: {k[len(p):]: v for k, v in w.items() if k.startswith(p)}
    x = w["embed"][np.asarray(tokens)]
    for i, layer in enumerate(config["layers"]):
        y = MIXERS[layer["type"]](centred_norm(x, w[f"l{i}.norm1"], eps), below(f"l{i}.mix."), layer["mixer"], eps)
        x = x + m * w[f"l{i}.ls1"] * y
        if layer.get("mlp"):
            x = x + m * w[f"l{i}.ls2"] * routed_ffn(centred_norm(x, w[f"l{i}.norm2"], eps), below(f"l{i}.mlp."), layer["mlp"])
        if layers_out is not None:
            layers_out.append(x)
    return centred_norm(x, w["final.norm"], eps) @ w["head"].T


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
