"""Plain, slow Logozen: one function per mechanism, one sequence at a time, no cache and no batching. The oracle of
tests/test_logozen.py; it shares no code with dlti_b200. Weights are a dict name -> tensor; everything runs in the dtype
of the inputs (float64 in the tests)."""
import math

import torch


def root_mean_square(x, eps):
    return torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def layer_norm(x, weight, eps):
    centred = x - x.mean(-1, keepdim=True)
    return centred / torch.sqrt((centred * centred).mean(-1, keepdim=True) + eps) * weight


def causal_conv(x, weight):
    """Per channel: y_t = sum_j weight[:, j] * x_(t - taps + 1 + j), zeros before the start."""
    taps = weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(weight[:, j] * padded[j:j + x.shape[0]] for j in range(taps))


def with_conv(h, weight):
    """The input convolution of a sublayer."""
    return h + causal_conv(h, weight)


def streams_in(xs, w_in):
    """xs [streams, T, d] -> what the sublayer's norm reads."""
    return sum(w_in[s] * xs[s] for s in range(len(xs)))


def streams_out(xs, y, mix, w_out):
    """New streams from the old ones (mix[from, to]) and the sublayer's output."""
    n = len(xs)
    return torch.stack([sum(mix[s, t] * xs[s] for s in range(n)) + w_out[t] * y for t in range(n)])


def rotate_pairs(x, base, dims):
    """x [T, ..., dim] at positions 0 .. T - 1: coordinates (2i, 2i+1) of the first `dims` turn by position * base^(-2i/dims)."""
    out = x.clone()
    for i in range(dims // 2):
        a = torch.arange(x.shape[0], dtype=torch.float64) * base ** (-2.0 * i / dims)
        c, s = (f(a).to(x.dtype).view(-1, *[1] * (x.dim() - 2)) for f in (torch.cos, torch.sin))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * c - v * s
        out[..., 2 * i + 1] = v * c + u * s
    return out


def attend(q, k, v, scale, sink):
    """q, k [T, H, d], v [T, H, dv], causal; sink [H]: one more term exp(sink) in every denominator, without a value."""
    T, H, _ = q.shape
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    later = torch.ones(T, T, dtype=torch.bool).triu(1)
    for h in range(H):
        s = (q[:, h] @ k[:, h].T * scale).masked_fill(later, -math.inf)
        top = torch.maximum(s.max(1).values, sink[h])[:, None]
        e = torch.exp(s - top)
        out[:, h] = e @ v[:, h] / (e.sum(1, keepdim=True) + torch.exp(sink[h] - top))
    return out


def latent_heads(q, down, gate, p, m, eps):
    """Projected rows (queries, latent | shared key part, gate numbers) -> head outputs [T, H * vdim]."""
    T, H = q.shape[0], m["heads"]
    q = q.view(T, H, m["dim"] + m["rot_dim"])
    q_plain, q_rot = q[..., :m["dim"]], q[..., m["dim"]:]
    c = down[:, :m["kv_rank"]]
    c = c / root_mean_square(c, eps) * p["dkv.norm"]
    k_rot = rotate_pairs(down[:, m["kv_rank"]:], m["rot"]["base"], m["rot"]["dims"])
    q_rot = rotate_pairs(q_rot, m["rot"]["base"], m["rot"]["dims"])
    k_plain = (c @ p["uk"].T).view(T, H, m["dim"])
    v = (c @ p["uv"].T).view(T, H, m["vdim"])
    k = torch.cat([k_plain, k_rot[:, None].expand(T, H, m["rot_dim"])], -1)
    o = attend(torch.cat([q_plain, q_rot], -1), k, v, m["scale"], p["sink"])
    return (o * torch.sigmoid(gate)[:, :, None]).reshape(T, -1)


def latent_attention(h, p, m, eps):
    return latent_heads(h @ p["q"].T, h @ p["dkv"].T, h @ p["g"].T, p, m, eps) @ p["o"].T


def log_sigmoid(z):
    return -torch.logaddexp(-z, torch.zeros_like(z))


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap)


def matrix_memory(q, k, v, log_in, log_forget):
    """q, k [T, heads, d], v [T, heads, dv], log gates [T, heads] -> [T, heads, dv]."""
    T, heads, d = q.shape
    S = torch.zeros(heads, d, v.shape[2], dtype=q.dtype)
    n = torch.zeros(heads, d, dtype=q.dtype)
    m = torch.zeros(heads, dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        m_new = torch.maximum(log_forget[t] + m, log_in[t])
        keep, add = torch.exp(log_forget[t] + m - m_new), torch.exp(log_in[t] - m_new)
        S = keep[:, None, None] * S + add[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + add[:, None] * k[t]
        m = m_new
        num = (S * q[t][:, :, None]).sum(1)
        den = torch.maximum((n * q[t]).sum(1).abs(), torch.exp(-m)) + 1e-6
        out[t] = num / den[:, None]
    return out


def mlstm(h, p, m, eps):
    T, heads = h.shape[0], m["heads"]
    q = (h @ p["q"].T).view(T, heads, m["dim"]) * m["dim"] ** -0.5
    k = (h @ p["k"].T).view(T, heads, m["dim"])
    v = (h @ p["v"].T).view(T, heads, m["vdim"])
    log_in = soft_cap(h @ p["i"].T + p["i.b"], m["gate_cap"])
    log_forget = log_sigmoid(soft_cap(h @ p["f"].T + p["f.b"], m["gate_cap"]))
    o = matrix_memory(q, k, v, log_in, log_forget)
    o = (o / root_mean_square(o, eps)).reshape(T, -1) * p["norm"]
    return (o * torch.sigmoid(h @ p["g"].T)) @ p["o"].T


def poly_norm(z, coef, eps):
    a, b, c, e = coef
    unit = lambda y: y / root_mean_square(y, eps)
    return a * unit(z) + b * unit(z * z) + c * unit(z * z * z) + e


def feed_forward(h, p, eps):
    return poly_norm(h @ p["up"].T, p["act"], eps) @ p["down"].T


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, after_layer=None):
    """Logits [T, vocab] of one sequence. after_layer: optional list that receives the sum of the streams after each layer."""
    eps = cfg["norm"]["eps"]
    x = weights["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    xs = torch.stack([x] * cfg["streams"])
    for i, layer in enumerate(cfg["layers"]):
        p = sub(weights, f"l{i}.")
        mixer = {"latent_attention": latent_attention, "mlstm": mlstm}[layer["type"]]
        parts = [(1, lambda h: mixer(h, sub(p, "mix."), layer["mixer"], eps))]
        if layer["mlp"] is not None:
            parts.append((2, lambda h: feed_forward(h, sub(p, "mlp."), eps)))
        for n, f in parts:
            h = layer_norm(streams_in(xs, p[f"hc{n}.in"]), p[f"norm{n}"], eps)
            y = f(with_conv(h, p[f"canon{n}"]))
            xs = streams_out(xs, y, p[f"hc{n}.mix"], p[f"hc{n}.out"])
        if after_layer is not None:
            after_layer.append(xs.sum(0))
    return layer_norm(xs.sum(0), weights["final.norm"], eps) @ weights["head"].T
