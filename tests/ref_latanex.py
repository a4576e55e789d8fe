"""Plain, slow Latanex: one function per mechanism, one sequence at a time, no cache and no batching. The oracle of
tests/test_latanex.py; it shares no code with dlti_b200. Weights are a dict name -> tensor; everything runs in the dtype
of the inputs (float64 in the tests)."""
import math

import torch


def dynamic_tanh(x, alpha, weight, bias):
    return torch.tanh(alpha * x) * weight + bias


def root_mean_square(x, eps):
    return torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def whole_norm(x, weight, eps):
    """One root mean square over all heads of a projection."""
    return x / root_mean_square(x, eps) * weight


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.logaddexp(z, torch.zeros_like(z))


def attend(q, k, v, scale, cap, window, sink):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: causal, at most `window` keys (0: all), scores capped softly; sink [H]: one more
    term exp(sink) in every denominator, without a value."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    hidden = (j > i) | ((i - j >= window) if window else torch.zeros(1, dtype=torch.bool))
    for h in range(H):
        s = q[:, h] @ k[:, h // rep].T * scale
        if cap:
            s = cap * torch.tanh(s / cap)
        s = s.masked_fill(hidden, -math.inf)
        top = torch.maximum(s.max(1).values, sink[h])[:, None]
        e = torch.exp(s - top)
        out[:, h] = e @ v[:, h // rep] / (e.sum(1, keepdim=True) + torch.exp(sink[h] - top))
    return out


def mix_values(v, first, share):
    return (1 - share) * v + share * first


def attention(h, p, m, eps, first):
    """first: a dict that lives for one forward pass; it keeps the values of the first layer that mixes."""
    T = h.shape[0]
    q, k, v = (h @ p[x].T + p[x + ".b"] for x in "qkv")
    q = whole_norm(q, p["q.norm"], eps).view(T, m["heads"], m["dim"])
    k = whole_norm(k, p["k.norm"], eps).view(T, m["kv_heads"], m["dim"])
    if m.get("v_mix"):
        if "v" in first:
            v = mix_values(v, first["v"], p["vmix"])
        else:
            first["v"] = v
    v = v.view(T, m["kv_heads"], m["vdim"])
    o = attend(q, k, v, m["scale"], m.get("softcap"), (m.get("mask") or {}).get("size") or 0, p["sink"])
    return o.reshape(T, -1) @ p["o"].T


def causal_conv(x, weight):
    """Per channel: y_t = sum_j weight[:, j] * x_(t - taps + 1 + j), zeros before the start."""
    taps = weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(weight[:, j] * padded[j:j + x.shape[0]] for j in range(taps))


def unit(x):
    return x / torch.sqrt((x * x).sum(-1, keepdim=True) + 1e-6)


def delta_rule(q, k, v, beta, decay):
    """q, k [T, heads, d], v [T, heads, dv], beta, decay [T, heads] -> [T, heads, dv]."""
    T, heads, d = q.shape
    S = torch.zeros(heads, d, v.shape[2], dtype=q.dtype)
    out = torch.zeros_like(v)
    for t in range(T):
        S = decay[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - (S * k[t][:, :, None]).sum(1))
        S = S + k[t][:, :, None] * u[:, None, :]
        out[t] = (S * q[t][:, :, None]).sum(1)
    return out


def step_decay(a, A_log, dt_bias):
    return torch.exp(-torch.exp(A_log) * softplus(a + dt_bias))


def delta(h, p, m, eps, first):
    T, heads, groups = h.shape[0], m["heads"], m["kv_heads"]
    q, k, v = (silu(causal_conv(h @ p[x].T, p[x + ".conv"])) for x in "qkv")
    q = unit(q.view(T, groups, m["dim"])) * m["dim"] ** -0.5
    k = unit(k.view(T, groups, m["dim"]))
    q, k = (x.repeat_interleave(heads // groups, 1) for x in (q, k))
    o = delta_rule(q, k, v.view(T, heads, m["vdim"]), sigmoid(h @ p["b"].T), step_decay(h @ p["a"].T, p["A_log"], p["dt_bias"]))
    o = o / root_mean_square(o, eps) * p["norm"] * silu(h @ p["g"].T).view(T, heads, m["vdim"])
    return o.reshape(T, -1) @ p["o"].T


def swiglu(h, p, prefix=""):
    return (silu(h @ p[prefix + "gate"].T) * (h @ p[prefix + "up"].T)) @ p[prefix + "down"].T


def clipped_expert(h, p, prefix, limit):
    g = torch.clamp(h @ p[prefix + "gate"].T, max=limit)
    u = torch.clamp(h @ p[prefix + "up"].T, -limit, limit)
    return (g * sigmoid(1.702 * g) * (u + 1)) @ p[prefix + "down"].T


def route(z, correction, top, groups, keep, scale):
    """Router logits of one token -> [(expert, weight)]."""
    s = sigmoid(z)
    c = (s + correction).tolist()
    n = len(c) // groups
    parts = [range(g * n, (g + 1) * n) for g in range(groups)]
    by_score = sorted(range(groups), key=lambda g: -sum(sorted((c[e] for e in parts[g]), reverse=True)[:2]))
    open_ = [e for g in by_score[:keep] for e in parts[g]]
    chosen = sorted(open_, key=lambda e: -c[e])[:top]
    total = sum(s[e] for e in chosen) + 1e-20
    return [(e, s[e] / total * scale) for e in chosen]


def experts(h, p, m):
    r = m["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    z = h @ p["router"].T
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in route(z[t], p["correction"], r["top"], g["count"], g["keep"], r["scale"]):
            out[t] += w * clipped_expert(h[t], p, f"e{e}.", m["expert"]["limit"])
    if m.get("shared"):
        out = out + clipped_expert(h, p, "shared.", m["shared"]["limit"])
    return out


def feed_forward(h, p, m):
    return experts(h, p, m) if m["kind"] == "moe" else swiglu(h, p)


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, after_layer=None):
    """Logits [T, vocab] of one sequence. after_layer: optional list that receives the residual after each layer."""
    eps = cfg["norm"]["eps"]
    norm = lambda x, p, name: dynamic_tanh(x, p[name + ".alpha"], p[name], p[name + ".b"])
    x = weights["embed"][torch.as_tensor(tokens)] * cfg["embedding"]["scale"]
    first = {}
    for i, layer in enumerate(cfg["layers"]):
        p = sub(weights, f"l{i}.")
        mixer = {"attention": attention, "delta": delta}[layer["type"]]
        x = x + norm(mixer(norm(x, p, "norm1"), sub(p, "mix."), layer["mixer"], eps, first), p, "norm1b")
        if layer["mlp"] is not None:
            x = x + norm(feed_forward(norm(x, p, "norm2"), sub(p, "mlp."), layer["mlp"]), p, "norm2b")
        if after_layer is not None:
            after_layer.append(x)
    return norm(x, weights, "final.norm") @ weights["head"].T * cfg["logit_scale"]
