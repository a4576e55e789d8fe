"""Plain, slow Ridazen: one function per mechanism, one sequence at a time, no cache and no batching. The oracle of
tests/test_ridazen.py; it shares no code with dlti_b200. Weights are a dict name -> tensor; everything runs in the dtype
of the inputs (float64 in the tests)."""
import math

import torch


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def rms_norm(x, weight, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * weight


def causal_conv(x, weight):
    """Per channel: y_t = sum_j weight[:, j] * x_(t - taps + 1 + j), zeros before the start."""
    taps = weight.shape[1]
    padded = torch.cat([torch.zeros(taps - 1, x.shape[1], dtype=x.dtype), x])
    return sum(weight[:, j] * padded[j:j + x.shape[0]] for j in range(taps))


def query_factor(p, coef, every):
    return 1 + coef * math.log((p + 1) // every + 1)


def distance_bucket(n, rows, far):
    """Row of a table of `rows` for distance n: one row per distance in the first half, then rows of growing width up to `far`."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half)))


def attend(q, k, v, scale, bias=None):
    """q [T, H, d], k [T, G, d], v [T, G, dv]: causal; bias [T, H]: added to the score at distance n."""
    T, H, _ = q.shape
    rep = H // k.shape[1]
    out = torch.zeros(T, H, v.shape[2], dtype=q.dtype)
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    for h in range(H):
        s = q[:, h] @ k[:, h // rep].T * scale
        if bias is not None:
            s = s + bias[(i - j).clamp(min=0), h]
        s = s.masked_fill(j > i, -math.inf)
        e = torch.exp(s - s.max(1, keepdim=True).values)
        out[:, h] = e @ v[:, h // rep] / e.sum(1, keepdim=True)
    return out


def attention(h, p, m, eps):
    T = h.shape[0]
    q, k, v = (h @ p[x].T for x in "qkv")
    if m.get("conv"):
        q, k, v = (causal_conv(y, p[x + ".conv"]) for x, y in zip("qkv", (q, k, v)))
    q = rms_norm(q.view(T, m["heads"], m["dim"]), p["q.norm"], eps)
    k = rms_norm(k.view(T, m["kv_heads"], m["dim"]), p["k.norm"], eps)
    if m.get("q_temp"):
        t = m["q_temp"]
        q = q * torch.tensor([query_factor(i, t["coef"], t["every"]) for i in range(T)], dtype=q.dtype)[:, None, None]
    bias = None
    if m.get("bias_max"):
        rel = p["rel"]
        bias = rel[[distance_bucket(n, rel.shape[0], m["bias_max"]) for n in range(T)]]
    o = attend(q, k, v.view(T, m["kv_heads"], m["vdim"]), m["scale"], bias).reshape(T, -1)
    return (o * sigmoid(h @ p["g"].T)) @ p["o"].T


def relu2_expert(h, p, prefix):
    u = torch.clamp(h @ p[prefix + "up"].T, min=0)
    return (u * u) @ p[prefix + "down"].T


def route(z, top):
    """Router logits of one token -> [(expert, weight)]."""
    z = z.tolist()
    chosen = sorted(range(len(z)), key=lambda e: -z[e])[:top]
    w = [math.exp(z[e] - z[chosen[0]]) for e in chosen]
    return [(e, x / sum(w)) for e, x in zip(chosen, w)]


def experts(h, p, m):
    z = h @ p["router"].T + p["router.b"]
    out = torch.zeros_like(h)
    for t in range(h.shape[0]):
        for e, w in route(z[t], m["router"]["top"]):
            out[t] += w * relu2_expert(h[t], p, f"e{e}.")
    if m.get("shared"):
        out = out + relu2_expert(h, p, "shared.") * sigmoid(h @ p["shared.sg"].T)
    return out


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def token_side(x, e, p, eps):
    """e: the token's own vector for this layer."""
    return rms_norm((gelu_tanh(x @ p["gate"].T) * e) @ p["proj"].T, p["norm"], eps)


def softcap(z, cap):
    return cap * torch.tanh(z / cap)


def running_order(n, loop):
    """[(layer, whether the embedding is added in front of it)]"""
    if not loop:
        return [(i, False) for i in range(n)]
    a, b = loop["start"], loop["stop"]
    order = [(i, False) for i in range(a)]
    for t in range(loop["times"]):
        order += [(i, t > 0 and i == a) for i in range(a, b)]
    return order + [(i, False) for i in range(b, n)]


def sub(weights, prefix):
    return {k[len(prefix):]: v for k, v in weights.items() if k.startswith(prefix)}


def forward(cfg, weights, tokens, after_layer=None):
    """Logits [T, vocab] of one sequence. after_layer: optional list that receives the residual after each layer run."""
    eps, mult = cfg["norm"]["eps"], cfg.get("residual_mult", 1.0)
    ids = torch.as_tensor(tokens)
    emb = weights["embed"][ids]
    x = emb
    for i, again in running_order(len(cfg["layers"]), cfg.get("loop")):
        layer, p = cfg["layers"][i], sub(weights, f"l{i}.")
        if again:
            x = x + emb
        x = x + mult * attention(rms_norm(x, p["norm1"], eps), sub(p, "mix."), layer["mixer"], eps)
        if layer["mlp"] is not None:
            x = x + mult * experts(rms_norm(x, p["norm2"], eps), sub(p, "mlp."), layer["mlp"])
        if cfg.get("token_side"):
            dim = cfg["token_side"]["dim"]
            x = x + mult * token_side(x, weights["side.embed"][ids][:, i * dim:(i + 1) * dim], sub(p, "side."), eps)
        if after_layer is not None:
            after_layer.append(x)
    z = rms_norm(x, weights["final.norm"], eps) @ weights["head"].T * cfg["logit_scale"]
    return softcap(z, cfg["logit_softcap"]) if cfg.get("logit_softcap") else z
