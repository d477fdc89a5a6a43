"""A plain, slow implementation of the Duzozen language model in numpy, one function per mechanism: the oracle of
tests/test_duzozen_*.py. It shares no code with the product path (its own weight access, its own loops); everything is
computed in float64 from the stored weights unless a test asks for another type.

weights: dict name -> array, in the tensor names of a checkpoint ("l0.mix.q", "l1.mlp.e3.up", ...)."""
from __future__ import annotations

import math

import numpy as np

_erf = np.vectorize(math.erf, otypes=[np.float64])


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def gelu_erf(z):
    return 0.5 * z * (1.0 + _erf(z / math.sqrt(2.0)))


def silu(z):
    return z / (1.0 + np.exp(-z))


def visible(i, j, size):
    """Whether position i sees position j; size None: every earlier position and itself."""
    return 0 <= i - j and (size is None or i - j < size)


def soft_cap(score, cap):
    return score if cap is None else cap * np.tanh(score / cap)


def attention(q, k, v, scale, cap, size, q_pos=None):
    """q [T, H, D], k [S, G, D], v [S, G, Dv]; query t sits at position q_pos[t] (default: the last T of S)."""
    T, H, D = q.shape
    S, G, _ = k.shape
    q_pos = range(S - T, S) if q_pos is None else q_pos
    out = np.zeros((T, H, v.shape[2]))
    for t, i in enumerate(q_pos):
        js = [j for j in range(S) if visible(i, j, size)]
        for h in range(H):
            g = h // (H // G)
            s = soft_cap(k[js, g] @ q[t, h] * scale, cap)
            p = np.exp(s - s.max())
            out[t, h] = (p / p.sum()) @ v[js, g]
    return out


def mix_values(v, v_first, lam):
    return (1.0 - lam) * v + lam * v_first


def route(logits, correction, top, count, keep):
    """One token's router logits [E] -> (chosen indices, their weights)."""
    e = np.exp(logits - logits.max())
    s = e / e.sum()
    choice = s + correction
    per = len(s) // count
    best = sorted(range(count), key=lambda g: (-choice[g * per:(g + 1) * per].max(), g))[:keep]
    allowed = [i for i in range(len(s)) if i // per in best]
    chosen = sorted(allowed, key=lambda i: (-choice[i], i))[:top]
    return chosen, [s[i] for i in chosen]


def dense_ff(w, p, h):
    return gelu_erf(h @ w[p + "up"].T) @ w[p + "down"].T


def expert_ff(w, p, h):
    return (silu(h @ w[p + "gate"].T) * (h @ w[p + "up"].T)) @ w[p + "down"].T


def moe_ff(w, p, h, mlp):
    r = mlp["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    out = np.zeros_like(h)
    for t in range(h.shape[0]):
        chosen, weights = route(w[p + "router"] @ h[t], w[p + "correction"], r["top"], groups["count"], groups["keep"])
        for i, s in zip(chosen, weights):
            out[t] += s * (h[t] if i >= r["experts"] else expert_ff(w, f"{p}e{i}.", h[t:t + 1])[0])
    return out


def mixer(w, p, h, m, v_first):
    """Returns the mixer's output and this layer's unmixed values."""
    T = h.shape[0]
    H, G = m["heads"], m["kv_heads"]
    q = (h @ w[p + "q"].T).reshape(T, H, m["dim"])
    k = (h @ w[p + "k"].T).reshape(T, G, m["dim"])
    v = own = (h @ w[p + "v"].T).reshape(T, G, m["vdim"])
    if m.get("v_mix") and v_first is not None:
        v = mix_values(v, v_first, float(w[p + "vmix"]))
    o = attention(q, k, v, m["scale"], m.get("softcap"), (m.get("mask") or {}).get("size"))
    return o.reshape(T, -1) @ w[p + "o"].T, own


def forward(cfg, weights, tokens, layers_out=None):
    """Logits [T, vocab] of a whole sequence; layers_out: a list that receives the residual stream after every layer."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = w["embed"][np.asarray(tokens)]
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        o, own = mixer(w, p + "mix.", rms_norm(x, w[p + "norm1"], eps), layer["mixer"], v_first)
        if layer["mixer"].get("v_mix") and v_first is None:
            v_first = own
        x = x + rms_norm(o, w[p + "norm1b"], eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            h = rms_norm(x, w[p + "norm2"], eps)
            y = dense_ff(w, p + "mlp.", h) if mlp["kind"] == "dense" else moe_ff(w, p + "mlp.", h, mlp)
            x = x + rms_norm(y, w[p + "norm2b"], eps)
        if layers_out is not None:
            layers_out.append(x.copy())
    return rms_norm(x, w["final.norm"], eps) @ w["head"].T


def greedy(cfg, weights, prompt, steps):
    toks = list(prompt)
    for _ in range(steps):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]
