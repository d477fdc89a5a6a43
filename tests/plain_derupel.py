"""A plain, slow implementation of the Derupel language model in numpy, one function per mechanism: the oracle of
tests/test_derupel_*.py. It shares no code with the product path; everything is computed in float64 from the stored
weights, sequences token by token, attention over whole prefixes.

weights: dict name -> array, in the tensor names of a checkpoint ("l0.mix.dq", "l1.mlp.e3.up", ...)."""
from __future__ import annotations

import numpy as np

from plain_lm import rms_norm, silu


def sigmoid(z):
    return 1.0 / (1.0 + np.exp(-z))


# ---------------------------------------------------------------- feed-forward
def squared_relu(z):
    return np.maximum(z, 0.0) ** 2


def dense_ff(w, p, h):
    return squared_relu(h @ w[p + "up"].T) @ w[p + "down"].T


def clamped_gate(gate, up, limit):
    """Gate bounded above, linear part bounded on both sides and shifted by one."""
    g, u = np.minimum(gate, limit), np.clip(up, -limit, limit)
    return g * sigmoid(1.702 * g) * (u + 1.0)


def expert_ff(w, p, h, limit):
    return clamped_gate(h @ w[p + "gate"].T, h @ w[p + "up"].T, limit) @ w[p + "down"].T


def route(logits, top):
    """One token's router logits [E] -> (chosen experts, their scores). (Scores have the order of the logits.)"""
    s = sigmoid(logits)
    chosen = sorted(range(len(s)), key=lambda i: (-logits[i], i))[:top]
    return chosen, [s[i] for i in chosen]


def moe_ff(w, p, h, mlp):
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, scores = route(w[p + "router"] @ h[t], mlp["router"]["top"])
        for i, s in zip(chosen, scores):
            out[t] += expert_ff(w, f"{p}e{i}.", (s * h[t])[None], mlp["expert"]["limit"])[0]
    if mlp.get("shared"):
        out += expert_ff(w, p + "shared.", h, mlp["shared"]["limit"])
    return out


# ---------------------------------------------------------------- mixers
def rotate(x, positions, base, dims):
    """x [T, ..., D]: neighbouring pairs of the first `dims` dimensions turn by position * base^(-2 i / dims)."""
    out = np.array(x, np.float64)
    for t, p in enumerate(positions):
        for i in range(dims // 2):
            a = p * float(base) ** (-2.0 * i / dims)
            u, v = out[t, ..., 2 * i].copy(), out[t, ..., 2 * i + 1].copy()
            out[t, ..., 2 * i] = u * np.cos(a) - v * np.sin(a)
            out[t, ..., 2 * i + 1] = v * np.cos(a) + u * np.sin(a)
    return out


def decayed_attention(q, k, v, decay, state=None):
    """Linear attention with one decay per head, one token after the other. q, k [T, H, D], v [T, H, Dv]; returns the
    outputs [T, H, Dv] and the state [H, D, Dv]."""
    T, H, D = q.shape
    S = np.zeros((H, D, v.shape[2])) if state is None else np.array(state, np.float64)
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        for h in range(H):
            S[h] = decay[h] * S[h] + np.outer(k[t, h], v[t, h])
            out[t, h] = S[h].T @ q[t, h]
    return out, S


def causal_attention(q, k, v, scale):
    """q [T, H, D], k [S, H, D], v [S, H, Dv]; the queries are the last T of the S positions."""
    T, H, _ = q.shape
    S = k.shape[0]
    out = np.zeros((T, H, v.shape[2]))
    for t in range(T):
        n = S - T + t + 1
        for h in range(H):
            s = k[:n, h] @ q[t, h] * scale
            e = np.exp(s - s.max())
            out[t, h] = (e / e.sum()) @ v[:n, h]
    return out


def lightning(w, p, h, m, eps):
    T, H = h.shape[0], m["heads"]
    q = silu(h @ w[p + "q"].T).reshape(T, H, m["dim"])
    k = silu(h @ w[p + "k"].T).reshape(T, H, m["dim"])
    v = silu(h @ w[p + "v"].T).reshape(T, H, m["vdim"])
    o, _ = decayed_attention(q, k, v, m["decay"])
    o = rms_norm(o.reshape(T, -1), w[p + "norm"], eps)
    return (o * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


def latent_attention(w, p, h, m, eps):
    T, H, d, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"]
    pos = range(T)
    q = (rms_norm(h @ w[p + "dq"].T, w[p + "dq.norm"], eps) @ w[p + "uq"].T).reshape(T, H, d + r)
    kv = h @ w[p + "dkv"].T
    c = rms_norm(kv[:, :m["kv_rank"]], w[p + "dkv.norm"], eps)
    rot = m["rot"]
    k_rot = rotate(kv[:, None, m["kv_rank"]:], pos, rot["base"], rot["dims"])  # one head's worth, shared by all
    q_rot = rotate(q[..., d:], pos, rot["base"], rot["dims"])
    k = np.concatenate([(c @ w[p + "uk"].T).reshape(T, H, d), np.repeat(k_rot, H, 1)], -1)
    v = (c @ w[p + "uv"].T).reshape(T, H, m["vdim"])
    o = causal_attention(np.concatenate([q[..., :d], q_rot], -1), k, v, m["scale"])
    return (o.reshape(T, -1) * sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T


MIXERS = {"lightning": lightning, "latent_attention": latent_attention}


# ---------------------------------------------------------------- the model
def forward(cfg, weights, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence; layers_out: a list that receives the residual stream after every layer."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + rms_norm(MIXERS[layer["type"]](w, p + "mix.", x, layer["mixer"], eps), w[p + "norm1"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            y = dense_ff(w, p + "mlp.", x) if mlp["kind"] == "dense" else moe_ff(w, p + "mlp.", x, mlp)
            x = x + rms_norm(y, w[p + "norm2"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg, weights, prompt, steps):
    toks = list(prompt)
    for _ in range(steps):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]
