"""A plain float64 restatement of the Malulorn design, one function per mechanism, whole sequences at once from position
0 (or from `pos0` where a mechanism reads the position).  It shares no code with the package: torch on the CPU only.
Weights are a dict name -> tensor; configurations are the dicts of config.json."""
import math

import torch

F64 = torch.float64


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, w, b, eps):
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * w + b


def silu(z):
    return z * torch.sigmoid(z)


def rotate_pairs(x, positions, base):
    """x [T, n], entry 2i with entry 2i+1, by the angle position * base^(-2i/n)."""
    out = x.clone()
    n = x.shape[1]
    for i in range(n // 2):
        a = positions.to(F64) * float(base) ** (-2.0 * i / n)
        u, v = x[:, 2 * i], x[:, 2 * i + 1]
        out[:, 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[:, 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def causal(T):
    return torch.triu(torch.ones(T, T, dtype=torch.bool), 1)


def query_temperature(position, coef, every):
    return 1.0 + coef * math.log(math.floor((position + 1) / every) + 1)


def softmax_plus_one(s, masked):
    """exp(s_j) / (1 + sum_j exp(s_j)) over the keys that are not masked."""
    s = s.masked_fill(masked, -math.inf)
    m = s.max(dim=-1, keepdim=True).values.clamp(min=0.0)
    e = torch.exp(s - m)
    return e / (torch.exp(-m) + e.sum(dim=-1, keepdim=True))


def attention(h, W, p, m):
    T, H, G, K, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ W[p + "q"].T).view(T, H, K)
    k = (h @ W[p + "k"].T).view(T, G, K)
    v = (h @ W[p + "v"].T).view(T, G, V)
    g = torch.sigmoid(h @ W[p + "g"].T)
    temp = torch.tensor([query_temperature(t, m["q_temp"]["coef"], m["q_temp"]["every"]) for t in range(T)], dtype=F64)
    out = torch.zeros(T, H, V, dtype=F64)
    for hd in range(H):
        kv = hd // (H // G)
        s = ((q[:, hd] * temp[:, None]) @ k[:, kv].T) * m["scale"]
        out[:, hd] = softmax_plus_one(s, causal(T)) @ v[:, kv] * g[:, hd:hd + 1]
    return out.reshape(T, H * V) @ W[p + "o"].T


def latent_attention(h, W, p, m, eps):
    """Keys and values are expanded from the latent for every position (the plain form)."""
    T, H, dn, dr, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ W[p + "q"].T).view(T, H, dn + dr)
    down = h @ W[p + "dkv"].T
    c = rms_unit(down[:, :rank], eps) * W[p + "dkv.norm"]
    k_rot = rotate_pairs(down[:, rank:], pos, m["rot"]["base"])
    key = (c @ W[p + "uk"].T).view(T, H, dn)
    val = (c @ W[p + "uv"].T).view(T, H, dv)
    out = torch.zeros(T, H, dv, dtype=F64)
    for hd in range(H):
        q_rot = rotate_pairs(q[:, hd, dn:], pos, m["rot"]["base"])
        s = (q[:, hd, :dn] @ key[:, hd].T + q_rot @ k_rot.T) * m["scale"]
        out[:, hd] = torch.softmax(s.masked_fill(causal(T), -math.inf), dim=-1) @ val[:, hd]
    return (out.reshape(T, H * dv) * torch.sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def gated(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(h, W, p, r):
    """Chosen experts [T, top], largest logit first, and the softmax over the chosen logits."""
    z = h @ W[p + "router"].T + W[p + "router.b"]
    v, idx = z.topk(r["top"], dim=-1)
    return idx, torch.softmax(v, dim=-1)


def experts(h, W, p, f):
    idx, wgt = route(h, W, p, f["router"])
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, a in zip(idx[t].tolist(), wgt[t]):
            out[t] += a * gated(h[t], W, f"{p}e{e}.")
    return out + gated(h, W, p + "shared.") if f.get("shared") else out


def inject(x, x0, W, t):
    """What stands before pass t of the loop."""
    return torch.cat([x, x0], dim=-1) @ W["loop.in"].T + W["loop.step"][t]


def layer(x, i, spec, W, eps):
    p = f"l{i}."
    h = layer_norm(x, W[p + "norm1"], W[p + "norm1.b"], eps)
    x = x + (attention(h, W, p + "mix.", spec["mixer"]) if spec["type"] == "attention" else latent_attention(h, W, p + "mix.", spec["mixer"], eps))
    if spec.get("mlp"):
        x = x + experts(layer_norm(x, W[p + "norm2"], W[p + "norm2.b"], eps), W, p + "mlp.", spec["mlp"])
    return x


def model(tokens, config, weights, capture=None):
    """tokens: list of ints, one whole sequence from position 0.  Returns logits [T, vocab] in float64."""
    W = {k: v.to(F64) for k, v in weights.items()}
    eps, layers, loop = config["norm"]["eps"], config["layers"], config.get("loop")
    x = x0 = W["embed"][torch.tensor(tokens)]
    runs = []                                       # (layer, the pass that starts with it or None)
    if loop:
        runs += [(i, None) for i in range(loop["start"])]
        for t in range(loop["times"]):
            runs += [(i, t if i == loop["start"] else None) for i in range(loop["start"], loop["stop"])]
        runs += [(i, None) for i in range(loop["stop"], len(layers))]
    else:
        runs = [(i, None) for i in range(len(layers))]
    for i, t in runs:
        if t is not None:
            x = inject(x, x0, W, t)
        x = layer(x, i, layers[i], W, eps)
        if capture is not None:
            capture.append(x.clone())
    return layer_norm(x, W["final.norm"], W["final.norm.b"], eps) @ W["head"].T
