"""Plain implementation of the Zogulorn decoder: whole sequences, float64, one function per mechanism, written from the
design's equations.  It shares no code with the package and is the oracle of the Zogulorn tests.

Notation: T tokens, width W.  ``tensors`` maps the checkpoint's names to float64 tensors.
"""
import math

import torch

F64 = torch.float64


def dynamic_tanh(x, w, name):
    """tanh(alpha x) * weight + bias; no statistic of the row."""
    return torch.tanh(w[name + ".alpha"] * x) * w[name] + w[name + ".b"]


def rms_unit(x, eps):
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


def gelu_tanh(x):
    return 0.5 * x * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (x + 0.044715 * x ** 3)))


def rotate_pairs(x, base, n):
    """x [T, heads, D]: channels 2i and 2i + 1 (i < n / 2) of the token at position p are turned by p * base^(-2i / n)."""
    out = x.clone()
    pos = torch.arange(x.shape[0], dtype=F64)
    for i in range(n // 2):
        a = (pos * base ** (-2.0 * i / n)).view(-1, 1)
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def block_mask(T, size):
    """[T, T]: query i sees key j <= i of its own block of ``size`` positions (None: of the whole sequence)."""
    i, j = torch.arange(T).view(-1, 1), torch.arange(T).view(1, -1)
    seen = j <= i
    return seen if size is None else seen & (i // size == j // size)


def softmax_rows(s, seen):
    s = s.masked_fill(~seen, -math.inf)
    e = torch.exp(s - s.max(dim=-1, keepdim=True).values)
    return e / e.sum(dim=-1, keepdim=True)


def short_conv(x, kernel):
    """x [T, C], kernel [C, taps] whose last column belongs to the current token; zeros before the start."""
    taps = kernel.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(kernel[:, j] * padded[j:j + x.shape[0]] for j in range(taps))


def _size(m):
    mask = m.get("mask")
    return None if mask is None else mask["size"]


def head_gate(h, w):
    """One number in (0, 1) per token and head."""
    return torch.sigmoid(h @ w["g"].T).unsqueeze(-1)


def rotary_attention(h, w, m):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    rot = lambda x: rotate_pairs(x, m["rot"]["base"], m["rot"]["dims"])
    q, k = rot((h @ w["q"].T).view(T, H, d)), rot((h @ w["k"].T).view(T, G, d))
    v = (h @ w["v"].T).view(T, G, dv)
    seen = block_mask(T, _size(m))
    o = torch.stack([softmax_rows(q[:, i] @ k[:, i // (H // G)].T * m["scale"], seen) @ v[:, i // (H // G)] for i in range(H)], 1)
    return (o * head_gate(h, w)).reshape(T, H * dv) @ w["o"].T


def channel_delta_rule(q, k, v, g, beta):
    """q, k, g [T, H, d], v [T, H, dv], beta [T, H]: row c of the state decays by g[.., c]; then the delta rule's write; then
    the answer to q."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F64)
    out = torch.zeros_like(v)
    for t in range(T):
        S = g[t].unsqueeze(-1) * S
        u = beta[t].unsqueeze(-1) * (v[t] - torch.einsum("hdv,hd->hv", S, k[t]))
        S = S + k[t].unsqueeze(-1) * u.unsqueeze(1)
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def decays(h, w, H, d):
    """[T, H, d] in (0, 1)."""
    z = softplus((h @ w["a1"].T) @ w["a2"].T + w["dt_bias"]).view(-1, H, d)
    return torch.exp(-torch.exp(w["A_log"]).view(1, H, 1) * z)


def channel_delta(h, w, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def branch(name):
        return silu(short_conv(h @ w[name].T, w[name + ".conv"]))

    unit = lambda x: x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)
    q, k = unit(branch("q").view(T, G, d)) * d ** -0.5, unit(branch("k").view(T, G, d))
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    o = channel_delta_rule(q, k, branch("v").view(T, H, dv), decays(h, w, H, d), torch.sigmoid(h @ w["b"].T))
    o = rms_unit(o, eps) * w["norm"]
    return (o.reshape(T, H * dv) * torch.sigmoid((h @ w["g1"].T) @ w["g2"].T)) @ w["o"].T


def difference(a1, a2, w, m, eps):
    """Two maps' outputs [T, H, dv] -> one."""
    lam = torch.exp((w["lq1"] * w["lk1"]).sum()) - torch.exp((w["lq2"] * w["lk2"]).sum()) + m["diff"]
    return rms_unit(a1 - lam * a2, eps) * (1.0 - m["diff"])


def keys_values(h, w, m):
    """The keys [T, G, 2, d] and values [T, G, dv] as a later layer may read them too."""
    T = h.shape[0]
    k = short_conv(h @ w["k"].T, w["k.conv"]).view(T, m["kv_heads"], 2, m["dim"])
    v = short_conv(h @ w["v"].T, w["v.conv"]).view(T, m["kv_heads"], m["vdim"])
    return k, v


def differential_attention(h, w, m, eps, kv):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = short_conv(h @ w["q"].T, w["q.conv"]).view(T, H, 2, d)
    k, v = kv
    seen = block_mask(T, _size(m))
    maps = [torch.stack([softmax_rows(q[:, i, j] @ k[:, i // (H // G), j].T * m["scale"], seen) @ v[:, i // (H // G)]
                         for i in range(H)], 1) for j in range(2)]
    o = difference(maps[0], maps[1], w, m, eps)
    return (o * head_gate(h, w)).reshape(T, H * dv) @ w["o"].T


def dense_ffn(h, w):
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def routed_ffn(h, w, m):
    z = h @ w["router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        best = torch.topk(z[t], m["router"]["top"])
        weights = torch.softmax(best.values, dim=0)
        for p, e in zip(weights, best.indices.tolist()):
            out[t] += p * (torch.clamp(h[t] @ w[f"e{e}.up"].T, min=0.0) ** 2 @ w[f"e{e}.down"].T)
    return out


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def forward(cfg, tensors, tokens, streams=None):
    """Logits [T, vocab] of one whole sequence.  ``streams``: a list that receives the stream after every layer."""
    eps = cfg["norm"]["eps"]
    x = tensors["embed"][torch.tensor(tokens)] * cfg["embedding"]["scale"]
    kept = {}
    for i, layer in enumerate(cfg["layers"]):
        t, m = sub(tensors, f"l{i}."), layer["mixer"]
        h, w = dynamic_tanh(x, t, "norm1"), sub(t, "mix.")
        if layer["type"] == "parallel":
            y = (m["left_scale"] * rotary_attention(h, sub(w, "left."), m["left"])
                 + m["right_scale"] * channel_delta(h, sub(w, "right."), m["right"], eps))
        elif layer["type"] == "attention":
            if m.get("kv_from") is None:
                kept[i] = keys_values(h, w, m)
            y = differential_attention(h, w, m, eps, kept[i if m.get("kv_from") is None else m["kv_from"]])
        else:
            raise ValueError(layer["type"])
        x = x + t["ls1"] * y
        f = layer.get("mlp")
        if f:
            h, w = dynamic_tanh(x, t, "norm2"), sub(t, "mlp.")
            x = x + t["ls2"] * (dense_ffn(h, w) if f["kind"] == "dense" else routed_ffn(h, w, f))
        if streams is not None:
            streams.append(x)
    return dynamic_tanh(x, tensors, "final.norm") @ tensors["head"].T


def greedy(cfg, tensors, tokens, steps):
    seq = list(tokens)
    for _ in range(steps):
        seq.append(int(forward(cfg, tensors, seq)[-1].argmax()))
    return seq[len(tokens):]
