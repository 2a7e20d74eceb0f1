"""Plain implementation of the layered designs (numpy, double precision), written from their equations: one function per mechanism, no
state carried between calls, no code shared with the library. Test infrastructure only.

Weights are a dict of tensor name -> array; shapes [out, in]; sequences are [tokens, width].
"""
from __future__ import annotations

import numpy as np


def sigmoid(z):
    return 0.5 * (1.0 + np.tanh(0.5 * np.asarray(z, np.float64)))


def silu(z):
    return z * sigmoid(z)


def rms_norm(x, w, eps):
    return x / np.sqrt(np.mean(x * x, axis=-1, keepdims=True) + eps) * w


def short_conv(u, w, b):
    """Causal convolution per channel: out[t, c] = b[c] + sum_k w[c, k] u[t - (taps - 1 - k), c], zeros before the start."""
    T, taps = len(u), w.shape[1]
    out = np.tile(np.asarray(b, np.float64), (T, 1))
    for k in range(taps):
        back = taps - 1 - k
        if back < T:
            out[back:] += w[:, k] * u[:T - back]
    return out


def mamba2(h, w, c, eps):
    heads, vdim, n, groups, parts = c["heads"], c["vdim"], c["state"], c["groups"], c["norm_groups"]
    inner, T = heads * vdim, len(h)
    p = h @ w["in"].T
    z, u, dt = p[:, :inner], p[:, inner:2 * inner + 2 * groups * n], p[:, 2 * inner + 2 * groups * n:]
    u = silu(short_conv(u, w["conv"], w["conv.b"]))
    x, B, C = u[:, :inner].reshape(T, heads, vdim), u[:, inner:inner + groups * n].reshape(T, groups, n), u[:, inner + groups * n:].reshape(T, groups, n)
    dt = np.logaddexp(0.0, dt + w["dt_bias"])
    y = np.zeros((T, heads, vdim))
    for k in range(heads):
        S, g = np.zeros((n, vdim)), k // (heads // groups)
        for t in range(T):
            S = np.exp(-np.exp(w["A_log"][k]) * dt[t, k]) * S + dt[t, k] * np.outer(B[t, g], x[t, k])
            y[t, k] = S.T @ C[t, g] + w["D"][k] * x[t, k]
    y = (y.reshape(T, inner) * silu(z)).reshape(T, parts, inner // parts)
    return rms_norm(y, np.reshape(w["norm"], (parts, -1)), eps).reshape(T, inner) @ w["o"].T


def hgrn2(h, w, c, eps):
    heads, dim, vdim, T = c["heads"], c["dim"], c["vdim"], len(h)
    q = silu(h @ w["q"].T).reshape(T, heads, dim)
    v = (h @ w["v"].T).reshape(T, heads, vdim)
    f = (w["lower"] + (1.0 - w["lower"]) * sigmoid(h @ w["f"].T + w["f.b"])).reshape(T, heads, dim)
    o = np.zeros((T, heads, vdim))
    for k in range(heads):
        S = np.zeros((dim, vdim))
        for t in range(T):
            S = f[t, k][:, None] * S + np.outer(1.0 - f[t, k], v[t, k])
            o[t, k] = q[t, k] @ S
    return rms_norm(o, w["norm"], eps).reshape(T, heads * vdim) @ w["o"].T


def visible(i, window, pool):
    """Of position i: the tokens it sees one by one, and the pooled blocks."""
    tokens = [j for j in range(i + 1) if i - j < window]
    blocks = [b for b in range(i // pool + 1) if (b + 1) * pool - 1 <= i - window]
    return tokens, blocks


def attention(h, w, c, eps):
    heads, kv, dim, vdim, T = c["heads"], c["kv_heads"], c["dim"], c["vdim"], len(h)
    window, pool = c["mask"]["size"], c["mask"]["pool"]
    q, k, v = (h @ w["q"].T).reshape(T, heads, dim), (h @ w["k"].T).reshape(T, kv, dim), (h @ w["v"].T).reshape(T, kv, vdim)
    gate = sigmoid(h @ w["g"].T)
    o = np.zeros((T, heads, vdim))
    for i in range(T):
        tokens, blocks = visible(i, window, pool)
        for a in range(heads):
            g = a // (heads // kv)
            keys = np.array([k[j, g] for j in tokens] + [k[b * pool:(b + 1) * pool, g].mean(0) for b in blocks])
            vals = np.array([v[j, g] for j in tokens] + [v[b * pool:(b + 1) * pool, g].mean(0) for b in blocks])
            s = keys @ q[i, a] * c["scale"]
            p = np.exp(s - s.max())
            o[i, a] = p / p.sum() @ vals * gate[i, a]
    return o.reshape(T, heads * vdim) @ w["o"].T


def feed_forward(h, gate, up, down):
    return (silu(h @ gate.T) * (h @ up.T)) @ down.T


def layer(x, w, spec, eps):
    """One parallel layer with two norms and gated residuals; ``w``: the layer's tensors without the layer prefix."""
    h = rms_norm(x, w["norm1"], eps)
    mix = {k[4:]: v for k, v in w.items() if k.startswith("mix.")}
    out = {"mamba2": mamba2, "hgrn2": hgrn2, "attention": attention}[spec["type"]](h, mix, spec["mixer"], eps) * sigmoid(h @ w["rg1"].T + w["rg1.b"])
    if spec["mlp"]:
        h = rms_norm(x, w["norm2"], eps)
        out = out + feed_forward(h, w["mlp.gate"], w["mlp.up"], w["mlp.down"]) * sigmoid(h @ w["rg2"].T + w["rg2.b"])
    return x + out


def lasosun(config, weights, tokens):
    """Logits [tokens, vocab] of a whole sequence."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    tokens = np.asarray(tokens)
    x = w["embed"][tokens] * config["embedding"]["scale"] + w["pos"][:len(tokens)]
    for i, spec in enumerate(config["layers"]):
        x = layer(x, {k[len(f"l{i}."):]: v for k, v in w.items() if k.startswith(f"l{i}.")}, spec, eps)
    return rms_norm(x, w["final.norm"], eps) @ w["embed"].T


# ---- Tosevik ---------------------------------------------------------------------------------------------------------------------------------
def unit(x, eps):
    """x divided by its root mean square over the last axis."""
    return rms_norm(x, 1.0, eps)


def dynamic_tanh(x, w, b, alpha):
    return np.tanh(alpha * x) * w + b


def rotate(x, positions, dims, base):
    """Rotary positions on the first ``dims`` entries of the last axis of x [tokens, heads, dim]; entry i turns with entry i + dims / 2."""
    half = dims // 2
    angle = np.asarray(positions, np.float64)[:, None] * base ** (-2.0 * np.arange(half) / dims)
    cos, sin = np.cos(angle)[:, None], np.sin(angle)[:, None]
    u, v = x[..., :half], x[..., half:dims]
    return np.concatenate([u * cos - v * sin, v * cos + u * sin, x[..., dims:]], -1)


def retention_state(q, k, v, decay):
    """o_t = S_t^T q_t with S_t = decay S_(t-1) + k_t v_t^T of one head, token by token."""
    S, o = np.zeros((k.shape[1], v.shape[1])), np.zeros((len(q), v.shape[1]))
    for t in range(len(q)):
        S = decay * S + np.outer(k[t], v[t])
        o[t] = S.T @ q[t]
    return o


def retention(h, w, c, eps):
    heads, dim, vdim, T = c["heads"], c["dim"], c["vdim"], len(h)
    q, k, v = (h @ w["q"].T).reshape(T, heads, dim), (h @ w["k"].T).reshape(T, heads, dim), (h @ w["v"].T).reshape(T, heads, vdim)
    q, k = (rotate(a, np.arange(T), c["rot"]["dims"], c["rot"]["base"]) for a in (q, k))
    o = np.stack([retention_state(q[:, a], k[:, a] * dim ** -0.5, v[:, a], c["decay"][a]) for a in range(heads)], 1)
    return (unit(o, eps).reshape(T, heads * vdim) * silu(h @ w["g"].T)) @ w["o"].T


def query_temperature(positions, coef, every):
    return 1.0 + coef * np.log(np.floor((np.asarray(positions) + 1) / every) + 1.0)


def distance_slopes(heads):
    return 2.0 ** (-8.0 * (np.arange(heads) + 1) / heads)


def sigmoid_attention(h, w, c, eps):
    heads, kv, dim, vdim, T = c["heads"], c["kv_heads"], c["dim"], c["vdim"], len(h)
    q, k = rms_norm(h @ w["q"].T, w["q.norm"], eps).reshape(T, heads, dim), rms_norm(h @ w["k"].T, w["k.norm"], eps).reshape(T, kv, dim)
    v = unit((h @ w["v"].T).reshape(T, kv, vdim), eps)
    if c.get("q_temp"):
        q = q * query_temperature(np.arange(T), c["q_temp"]["coef"], c["q_temp"]["every"])[:, None, None]
    back = np.arange(T)[:, None] - np.arange(T)[None, :]
    o = np.zeros((T, heads, vdim))
    for a in range(heads):
        g = a // (heads // kv)
        score = q[:, a] @ k[:, g].T * c["scale"] - distance_slopes(heads)[a] * back + w["pb"][a]
        o[:, a] = np.where(back >= 0, sigmoid(score), 0.0) @ v[:, g]
    return o.reshape(T, heads * vdim) @ w["o"].T


def part(w, prefix):
    return {k[len(prefix):]: v for k, v in w.items() if k.startswith(prefix)}


def side_by_side(h, w, c, eps):
    left = sigmoid_attention(h, part(w, "left."), c["left"], eps)
    right = retention(h, part(w, "right."), c["right"], eps)
    return 0.5 * (rms_norm(left, w["left.out"], eps) + rms_norm(right, w["right.out"], eps))


def route(z, c):
    """Of one token's router logits: the chosen experts and their weights."""
    s = np.exp(z - z.max())
    s /= s.sum()
    groups = np.arange(len(s)).reshape(c["groups"]["count"], -1)
    best = groups[np.argsort(-s[groups].max(1), kind="stable")[:c["groups"]["keep"]]].ravel()
    chosen = best[np.argsort(-s[best], kind="stable")[:c["top"]]]
    return chosen, s[chosen] * c["scale"]


def experts(h, w, c):
    out = np.zeros_like(h)
    for t in range(len(h)):
        for e, weight in zip(*route(w["router"] @ h[t], c["router"])):
            out[t] += weight * feed_forward(h[t], w[f"e{e}.gate"], w[f"e{e}.up"], w[f"e{e}.down"])
    return out + sigmoid(h @ w["shared.sg"].T) * feed_forward(h, w["shared.gate"], w["shared.up"], w["shared.down"])


def tosevik_stream(config, weights, tokens):
    """The residual stream after every layer [layers, tokens, width] - each after its depth average - and the logits [tokens, vocab]."""
    w = {k: np.asarray(v, np.float64) for k, v in weights.items()}
    eps = config["norm"]["eps"]
    norm = lambda x, name: dynamic_tanh(x, w[name], w[name + ".b"], w[name + ".alpha"])
    x = norm(w["embed"][np.asarray(tokens)], "embed.norm")
    results, stream = [x], []
    for i, spec in enumerate(config["layers"]):
        p = f"l{i}."
        x = x + {"retention": retention, "parallel": side_by_side}[spec["type"]](norm(x, p + "norm1"), part(w, p + "mix."), spec["mixer"], eps)
        if spec["mlp"]:
            x = x + experts(norm(x, p + "norm2"), part(w, p + "mlp."), spec["mlp"])
        results.append(x)
        x = sum(a * r for a, r in zip(w[p + "dwa"], results))
        stream.append(x)
    return np.stack(stream), norm(x, "final.norm") @ w["head"].T


def tosevik(config, weights, tokens):
    return tosevik_stream(config, weights, tokens)[1]
