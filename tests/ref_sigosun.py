"""Plain, slow Sigosun: one function per mechanism, one sequence at a time, no cache and no batching. The oracle of
tests/test_sigosun_*.py; it shares no code with dlti_b200. Weights are a dict name -> tensor; everything runs in the
dtype of the inputs (float64 in the tests)."""
import math

import torch


def rms_norm(x, weight, eps, one_plus=False):
    """x / sqrt(mean x^2 + eps), times `weight` (or 1 + weight)."""
    y = x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)
    return y * (1 + weight) if one_plus else y * weight


def rotate_pairs(x, positions, base, dims):
    """x [T, heads, dim]: coordinates (2i, 2i+1) of the first `dims` turn by position * base^(-2i/dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = positions.to(torch.float64) * base ** (-2.0 * i / dims)
        c, s = torch.cos(a).to(x.dtype)[:, None], torch.sin(a).to(x.dtype)[:, None]
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def visible(i, j, chunk):
    """May position i look at position j?"""
    return j <= i and (chunk is None or i // chunk == j // chunk)


def softmax_attention(q, k, v, scale, chunk):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    for i in range(T):
        js = [j for j in range(T) if visible(i, j, chunk)]
        kk, vv = k[js], v[js]
        for h in range(H):
            w = torch.softmax((kk[:, h // rep] @ q[i, h]) * scale, dim=0)
            out[i, h] = w @ vv[:, h // rep]
    return out


def attention_keys_values(h, p, m, eps):
    T = h.shape[0]
    k = (h @ p["k"].T).view(T, m["kv_heads"], m["dim"])
    v = (h @ p["v"].T).view(T, m["kv_heads"], m["vdim"])
    k = rms_norm(k, p["k.norm"], eps)
    return rotate_pairs(k, torch.arange(T), m["rot"]["base"], m["rot"]["dims"]), v


def attention(h, p, m, eps, kv=None):
    """Returns (output, (keys, values)); kv = another layer's keys and values to use instead of own ones."""
    T = h.shape[0]
    q = (h @ p["q"].T).view(T, m["heads"], m["dim"])
    q = rms_norm(q, p["q.norm"], eps)
    q = rotate_pairs(q, torch.arange(T), m["rot"]["base"], m["rot"]["dims"])
    if kv is None:
        kv = attention_keys_values(h, p, m, eps)
    o = softmax_attention(q, kv[0], kv[1], m["scale"], m["mask"]["size"])
    o = o * torch.sigmoid(h @ p["g"].T)[:, :, None]
    return o.reshape(T, -1) @ p["o"].T, kv


def causal_conv(x, weight, bias):
    """Per channel: y_t = bias + sum_k weight[:, k] * x_(t - taps + 1 + k), zeros before the start."""
    taps = weight.shape[1]
    y = torch.zeros_like(x)
    for t in range(x.shape[0]):
        acc = bias.clone()
        for k in range(taps):
            src = t - taps + 1 + k
            if src >= 0:
                acc = acc + weight[:, k] * x[src]
        y[t] = acc
    return y


def silu(x):
    return x * torch.sigmoid(x)


def ssd_recurrence(x, B, C, dt, A_log, D):
    """x [T, heads, P], B, C [T, G, N], dt [T, heads] (after softplus) -> y [T, heads, P]."""
    T, heads, P = x.shape
    G, N = B.shape[1:]
    y = torch.zeros_like(x)
    for h in range(heads):
        g = h // (heads // G)
        S = torch.zeros(N, P, dtype=x.dtype)
        for t in range(T):
            S = math.e ** (-torch.exp(A_log[h]) * dt[t, h]) * S + dt[t, h] * torch.outer(B[t, g], x[t, h])
            y[t, h] = C[t, g] @ S + D[h] * x[t, h]
    return y


def mamba2(h, p, m, eps):
    T = h.shape[0]
    heads, P, N, G = m["heads"], m["vdim"], m["state"], m["groups"]
    inner = heads * P
    z, xbc, dt = torch.split(h @ p["in"].T, [inner, inner + 2 * G * N, heads], dim=1)
    xbc = silu(causal_conv(xbc, p["conv"], p["conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=1)
    dt = torch.logaddexp(dt + p["dt_bias"], torch.zeros_like(dt))
    y = ssd_recurrence(x.reshape(T, heads, P), B.reshape(T, G, N), C.reshape(T, G, N), dt, p["A_log"], p["D"])
    y = (y.reshape(T, inner) * silu(z)).view(T, m["norm_groups"], -1)
    y = y / torch.sqrt((y * y).mean(-1, keepdim=True) + eps)
    return (y.reshape(T, inner) * p["norm"]) @ p["o"].T


def decay_recurrence(q, k, v, decay):
    """q, k [T, heads, d], v [T, heads, dv], one decay per head -> [T, heads, dv]."""
    T, heads, d = q.shape
    o = torch.zeros_like(v)
    for h in range(heads):
        S = torch.zeros(d, v.shape[2], dtype=q.dtype)
        for t in range(T):
            S = decay[h] * S + torch.outer(k[t, h], v[t, h])
            o[t, h] = q[t, h] @ S
    return o


def lightning(h, p, m, eps):
    T = h.shape[0]
    q = silu(h @ p["q"].T).view(T, m["heads"], m["dim"])
    k = silu(h @ p["k"].T).view(T, m["heads"], m["dim"])
    v = silu(h @ p["v"].T).view(T, m["heads"], m["vdim"])
    o = decay_recurrence(q, k, v, m["decay"]).reshape(T, -1)
    return (rms_norm(o, p["norm"], eps) * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


def squared_relu_mlp(h, p):
    return torch.relu(h @ p["up"].T).square() @ p["down"].T


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, after_layer=None):
    """Logits [T, vocab] of one sequence. after_layer: optional list that receives the residual after each layer."""
    eps = cfg["norm"]["eps"]
    x = weights["embed"][torch.as_tensor(tokens)]
    kvs = {}
    for i, layer in enumerate(cfg["layers"]):
        m, p = layer["mixer"], sub(weights, f"l{i}.mix.")
        if layer["type"] == "attention":
            src = m.get("kv_from")
            y, kvs[i] = attention(x, p, m, eps, None if src is None else kvs[src])
        else:
            y = {"mamba2": mamba2, "lightning": lightning}[layer["type"]](x, p, m, eps)
        x = x + rms_norm(y, weights[f"l{i}.norm1"], eps, one_plus=True)
        if layer["mlp"] is not None:
            y = squared_relu_mlp(x, sub(weights, f"l{i}.mlp."))
            x = x + rms_norm(y, weights[f"l{i}.norm2"], eps, one_plus=True)
        if after_layer is not None:
            after_layer.append(x)
    return rms_norm(x, weights["final.norm"], eps, one_plus=True) @ weights["head"].T
