"""A plain float64 restatement of the Lukupel design, one function per mechanism, written token by token wherever a
loop is the plainest form.  It shares no code with the package: torch on the CPU only.  Weights are a dict
name -> tensor; configurations are the dicts of config.json.  Every function takes a whole sequence from position 0."""
import math

import torch

F64 = torch.float64


def w64(W, name):
    return W[name].to(F64)


# ---------------------------------------------------------------------------------------------- norms
def unit_rms(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def rms_norm(x, w, eps):
    return unit_rms(x, eps) * w


# ---------------------------------------------------------------------------------------------- rotation
def frequencies(rot):
    """One frequency per pair; a linear scaling slows every pair down by the same factor."""
    dims, base = rot["dims"], float(rot["base"])
    factor = float((rot.get("scaling") or {}).get("factor", 1.0))
    return [base ** (-2.0 * i / dims) / factor for i in range(dims // 2)]


def rotate(vec, position, freqs):
    """vec [n]: entries i and i + len(freqs) turn by position * freqs[i], the rest stay."""
    out = vec.clone()
    half = len(freqs)
    for i, f in enumerate(freqs):
        c, s = math.cos(position * f), math.sin(position * f)
        out[i] = vec[i] * c - vec[i + half] * s
        out[i + half] = vec[i + half] * c + vec[i] * s
    return out


# ---------------------------------------------------------------------------------------------- attention inside chunks
def heads_rotated_then_normed(x, heads, dim, rot, eps):
    T = x.shape[0]
    x = x.view(T, heads, dim).clone()
    if rot and rot.get("dims"):
        f = frequencies(rot)
        for t in range(T):
            for h in range(heads):
                x[t, h] = rotate(x[t, h], t, f)
    return unit_rms(x, eps)


def visible_from(position, size):
    """First position that the query at `position` sees: the start of its chunk (no size: the start of the sequence)."""
    return (position // size) * size if size else 0


def chunk_attention(h, W, p, c, eps):
    T, H, G, K, V = h.shape[0], c["heads"], c["kv_heads"], c["dim"], c["vdim"]
    q = heads_rotated_then_normed(h @ w64(W, p + "q").T, H, K, c.get("rot"), eps)
    k = heads_rotated_then_normed(h @ w64(W, p + "k").T, G, K, c.get("rot"), eps)
    v = (h @ w64(W, p + "v").T).view(T, G, V)
    size = (c.get("mask") or {}).get("size")
    out = torch.zeros(T, H, V, dtype=F64)
    for i in range(T):
        lo = visible_from(i, size)
        for hd in range(H):
            g = hd // (H // G)
            s = (k[lo:i + 1, g] @ q[i, hd]) * c["scale"]
            w = torch.exp(s - s.max())
            w = w / w.sum()
            out[i, hd] = (w[:, None] * v[lo:i + 1, g]).sum(dim=0)
    return out.reshape(T, H * V) @ w64(W, p + "o").T


# ---------------------------------------------------------------------------------------------- matrix memory
def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def log_gates(h, W, p, cap):
    """Logarithms of the input gate and of the forget gate, [T, heads] each."""
    i = soft_cap(h @ w64(W, p + "i").T + w64(W, p + "i.b"), cap)
    z = soft_cap(h @ w64(W, p + "f").T + w64(W, p + "f.b"), cap)
    return i, -torch.log1p(torch.exp(-z))


def matrix_memory(q, k, v, log_i, log_f, lose=None):
    """One head, token by token: q, k [T, K] (q already scaled), v [T, V], the two log gates [T] -> read-outs [T, V].
    lose = (token, "S" | "n" | "m"): a planted mistake, that part of the state is gone before the token."""
    T, K, V = q.shape[0], q.shape[1], v.shape[1]
    S, n, m = torch.zeros(K, V, dtype=F64), torch.zeros(K, dtype=F64), 0.0
    out = torch.zeros(T, V, dtype=F64)
    for t in range(T):
        if lose and lose[0] == t:
            S, n, m = S * (lose[1] != "S"), n * (lose[1] != "n"), m * (lose[1] != "m")
        i, f = float(log_i[t]), float(log_f[t])
        new = max(f + m, i)
        keep, put = math.exp(f + m - new), math.exp(i - new)
        S = keep * S + put * torch.outer(k[t], v[t])
        n = keep * n + put * k[t]
        m = new
        out[t] = (S.T @ q[t]) / (max(abs(float(n @ q[t])), math.exp(-m)) + 1e-6)
    return out


def mlstm(h, W, p, c, eps, lose=None):
    T, H, K, V = h.shape[0], c["heads"], c["dim"], c["vdim"]
    q = (h @ w64(W, p + "q").T).view(T, H, K) * K ** -0.5
    k = (h @ w64(W, p + "k").T).view(T, H, K)
    v = (h @ w64(W, p + "v").T).view(T, H, V)
    log_i, log_f = log_gates(h, W, p, c["gate_cap"])
    o = torch.stack([matrix_memory(q[:, a], k[:, a], v[:, a], log_i[:, a], log_f[:, a], lose) for a in range(H)], dim=1)
    o = unit_rms(o, eps).reshape(T, H * V) * w64(W, p + "norm") * torch.sigmoid(h @ w64(W, p + "g").T)
    return o @ w64(W, p + "o").T


# ---------------------------------------------------------------------------------------------- feed-forward
def dense_ff(h, W, p):
    u = torch.clamp(h @ w64(W, p + "up").T, min=0.0)
    return (u * u) @ w64(W, p + "down").T


# ---------------------------------------------------------------------------------------------- the model
def owner(layers, i):
    """The layer whose tensors layer i uses."""
    while layers[i].get("weights_of") is not None:
        i = layers[i]["weights_of"]
    return i


def model(tokens, cfg, W, capture=None):
    """Logits [T, vocab] of a whole sequence.  `capture` (a list) receives the residual stream after every layer."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = w64(W, "embed")[torch.tensor(tokens)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p, c = f"l{owner(cfg['layers'], i)}.", layer["mixer"]
        y = mlstm(x, W, p + "mix.", c, eps) if layer["type"] == "mlstm" else chunk_attention(x, W, p + "mix.", c, eps)
        x = x + mult * rms_norm(y, w64(W, p + "norm1"), eps)
        if layer.get("mlp"):
            x = x + mult * rms_norm(dense_ff(x, W, p + "mlp."), w64(W, p + "norm2"), eps)
        if capture is not None:
            capture.append(x)
    z = rms_norm(x, w64(W, "final.norm"), eps) @ w64(W, "embed").T
    return soft_cap(z, cfg["logit_softcap"])
