"""Plain implementation of the Zanivik decoder: whole sequences, float64, one function per mechanism, written from the
design's equations.  It shares no code with the package and is the oracle of the Zanivik tests.

Notation: T tokens, width W.  ``tensors`` maps the checkpoint's names to float64 tensors.
"""
import math

import torch

F64 = torch.float64


def rms_unit(x, eps):
    """x / sqrt(mean(x^2) + eps) over the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def layer_norm(x, gain, eps):
    """Mean off, divided by the square root of the mean squared deviation plus eps, times the gain; no bias."""
    d = x - x.mean(dim=-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(dim=-1, keepdim=True) + eps) * gain


def silu(x):
    return x * torch.sigmoid(x)


def softplus(x):
    return torch.clamp(x, min=0.0) + torch.log1p(torch.exp(-x.abs()))


def gelu(x):
    return 0.5 * x * (1.0 + torch.erf(x / math.sqrt(2.0)))


def frequencies(rot):
    """The rotation's frequencies, one per pair of channels, with the wavelength bands of ``rot['scaling']``."""
    n = rot["dims"]
    out = []
    for i in range(n // 2):
        f = rot["base"] ** (-2.0 * i / n)
        s = rot.get("scaling")
        if s:
            wave = 2.0 * math.pi / f
            if wave > s["original"] / s["low"]:
                f = f / s["factor"]
            elif wave >= s["original"] / s["high"]:
                keep = (s["original"] / wave - s["low"]) / (s["high"] - s["low"])
                f = (1.0 - keep) * f / s["factor"] + keep * f
        out.append(f)
    return out


def rotate_halves(x, rot):
    """x [T, heads, D]: of the first n = rot['dims'] channels, channel i and channel i + n / 2 of the token at position p
    are turned by p * f_i; the others pass."""
    T, n = x.shape[0], rot["dims"]
    ang = torch.arange(T, dtype=F64).view(-1, 1) * torch.tensor(frequencies(rot), dtype=F64)
    c, s = torch.cos(ang).unsqueeze(1), torch.sin(ang).unsqueeze(1)
    a, b = x[..., :n // 2], x[..., n // 2:n]
    return torch.cat([a * c - b * s, b * c + a * s, x[..., n:]], dim=-1)


def window_mask(T, size):
    d = torch.arange(T).view(-1, 1) - torch.arange(T).view(1, -1)
    return (d >= 0) & (d < size) if size is not None else d >= 0


def attend(q, k, v, scale, visible, sink=None, head_factor=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H * dv].  ``sink`` [H]: exp(sink) joins the denominator.
    ``head_factor`` [H] multiplies the scores."""
    T, H = q.shape[:2]
    G = k.shape[1]
    out = []
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T) * scale
        if head_factor is not None:
            s = s * head_factor[h]
        s = s.masked_fill(~visible, -math.inf)
        m = s.max(dim=-1, keepdim=True).values
        if sink is not None:
            m = torch.clamp(m, min=float(sink[h]))
        e = torch.exp(s - m)
        den = e.sum(dim=-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - m)
        out.append((e / den) @ v[:, g])
    return torch.cat(out, dim=-1)


def sink_attention(h, w, m, eps):
    """Attention whose queries and keys are divided by their root mean square after the rotation, with a sink and a gate."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = (h @ w["q"].T).view(T, H, d)
    k = (h @ w["k"].T).view(T, G, d)
    v = (h @ w["v"].T).view(T, G, dv)
    q, k = rms_unit(rotate_halves(q, m["rot"]), eps), rms_unit(rotate_halves(k, m["rot"]), eps)
    o = attend(q, k, v, m["scale"], window_mask(T, (m.get("mask") or {}).get("size")), sink=w["sink"])
    return (o * torch.sigmoid(h @ w["g"].T)) @ w["o"].T


def shared_kv_attention(h, w, m, eps):
    """Attention whose values are the key projection itself; gains on queries and keys before the rotation; a factor per
    head on the scores."""
    T = h.shape[0]
    H, G, d = m["heads"], m["kv_heads"], m["dim"]
    q = (h @ w["q"].T).view(T, H, d)
    k = (h @ w["k"].T).view(T, G, d)
    v = k
    q, k = rms_unit(q, eps) * w["q.norm"], rms_unit(k, eps) * w["k.norm"]
    q, k = rotate_halves(q, m["rot"]), rotate_halves(k, m["rot"])
    o = attend(q, k, v, m["scale"], window_mask(T, (m.get("mask") or {}).get("size")), head_factor=w["temp"])
    return o @ w["o"].T


def short_conv(x, kernel, bias=None):
    """x [T, C], kernel [C, taps] whose last column belongs to the current token; zeros before the start."""
    T, taps = x.shape[0], kernel.shape[1]
    out = torch.zeros_like(x)
    for t in range(T):
        for j in range(taps):
            s = t - (taps - 1 - j)
            if s >= 0:
                out[t] += kernel[:, j] * x[s]
    return out if bias is None else out + bias


def delta_rule(q, k, v, g, beta):
    """q, k [T, H, d], v [T, H, dv], g, beta [T, H]: the state decays, takes in what it does not yet say about k, answers q."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[2], dtype=F64)
    out = torch.zeros_like(v)
    for t in range(T):
        for h in range(H):
            S[h] = g[t, h] * S[h]
            u = beta[t, h] * (v[t, h] - S[h].T @ k[t, h])
            S[h] = S[h] + torch.outer(k[t, h], u)
            out[t, h] = S[h].T @ q[t, h]
    return out


def gated_delta(h, w, m, eps):
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]

    def branch(name):
        return silu(short_conv(h @ w[name].T, w[name + ".conv"]))

    q, k, v = branch("q").view(T, G, d), branch("k").view(T, G, d), branch("v").view(T, H, dv)
    q = q / torch.sqrt((q * q).sum(-1, keepdim=True) + 1e-6) * d ** -0.5
    k = k / torch.sqrt((k * k).sum(-1, keepdim=True) + 1e-6)
    q, k = q.repeat_interleave(H // G, dim=1), k.repeat_interleave(H // G, dim=1)
    beta = torch.sigmoid(h @ w["b"].T)
    g = torch.exp(-torch.exp(w["A_log"]) * softplus(h @ w["a"].T + w["dt_bias"]))
    o = delta_rule(q, k, v, g, beta)
    o = rms_unit(o, eps) * w["norm"]
    o = o.reshape(T, H * dv) * silu(h @ w["g"].T)
    return o @ w["o"].T


def state_space(x, B, C, dt, A, D):
    """x [T, H, P], B, C [T, H, N], dt [T, H], A, D [H]: S <- exp(A dt) S + dt B x^T, y = S^T C + D x."""
    T, H, P = x.shape
    S = torch.zeros(H, B.shape[2], P, dtype=F64)
    y = torch.zeros_like(x)
    for t in range(T):
        for h in range(H):
            S[h] = torch.exp(A[h] * dt[t, h]) * S[h] + dt[t, h] * torch.outer(B[t, h], x[t, h])
            y[t, h] = S[h].T @ C[t, h] + D[h] * x[t, h]
    return y


def mamba2(h, w, m, eps):
    T = h.shape[0]
    H, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * P
    z, xbc, dt = torch.split(h @ w["in"].T, [inner, inner + 2 * G * N, H], dim=-1)
    xbc = silu(short_conv(xbc, w["conv"], w["conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=-1)
    x = x.reshape(T, H, P)
    B = B.reshape(T, G, N).repeat_interleave(H // G, dim=1)
    C = C.reshape(T, G, N).repeat_interleave(H // G, dim=1)
    y = state_space(x, B, C, softplus(dt + w["dt_bias"]), -torch.exp(w["A_log"]), w["D"]).reshape(T, inner)
    y = y * silu(z)
    y = rms_unit(y.view(T, m["norm_groups"], -1), eps).reshape(T, inner) * w["norm"]
    return y @ w["o"].T


def sub(tensors, prefix):
    return {k[len(prefix):]: v for k, v in tensors.items() if k.startswith(prefix)}


def mixer(kind, h, w, m, eps):
    left, right = sub(w, "left."), sub(w, "right.")
    if kind == "parallel":
        return (m["left_scale"] * sink_attention(h, left, m["left"], eps)
                + m["right_scale"] * gated_delta(h, right, m["right"], eps))
    if kind == "parallel_2":
        a = rms_unit(shared_kv_attention(h, left, m["left"], eps), eps) * left["out"]
        b = rms_unit(mamba2(h, right, m["right"], eps), eps) * right["out"]
        return 0.5 * (a + b)
    raise ValueError(kind)


def dense_ffn(h, w):
    return gelu(h @ w["up"].T) @ w["down"].T


def forward(cfg, tensors, tokens, streams=None):
    """Logits [T, vocab] of one whole sequence.  ``streams``: a list that receives the stream after every layer."""
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    x = tensors["embed"][torch.tensor(tokens)]
    for i, layer in enumerate(cfg["layers"]):
        t = sub(tensors, f"l{i}.")
        y = mixer(layer["type"], layer_norm(x, t["norm1"], eps), sub(t, "mix."), layer["mixer"], eps)
        x = x + mult * layer_norm(y, t["norm1b"], eps) * t["ls1"]
        if layer.get("mlp"):
            y = dense_ffn(layer_norm(x, t["norm2"], eps), sub(t, "mlp."))
            x = x + mult * layer_norm(y, t["norm2b"], eps) * t["ls2"]
        if streams is not None:
            streams.append(x)
    return layer_norm(x, tensors["final.norm"], eps) @ tensors["head"].T


def greedy(cfg, tensors, tokens, steps):
    seq = list(tokens)
    for _ in range(steps):
        seq.append(int(forward(cfg, tensors, seq)[-1].argmax()))
    return seq[len(tokens):]
