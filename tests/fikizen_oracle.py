"""Slow, plain restatement of the Fikizen decoder for the tests: one function per mechanism, whole sequences
at once, no cache, no batching, nothing imported from the package under test.

Notation: T tokens, D channels of the residual stream, `<.>` a mean over the last axis; arithmetic in the dtype
of the weights handed in (float64 in most tests)."""
import math

import torch


def rms_unit(x, eps):
    """x / sqrt(<x^2> + eps)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit(x):
    """x / sqrt(sum x^2 + 1e-6)."""
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + 1e-6)


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


def silu(z):
    return z * sigmoid(z)


def softplus(z):
    return torch.log1p(torch.exp(-z.abs())) + z.clamp(min=0)


def xielu(z, p, q):
    """softplus(p) z^2 + z / 2 above zero, (1/2 + softplus(q)) (e^z - 1 - z) + z / 2 below."""
    below = (0.5 + softplus(q)) * (torch.expm1(z.clamp(max=0)) - z)
    return torch.where(z > 0, softplus(p) * z * z, below) + z / 2


def rotate_halves(x, pos, base, dims):
    """x [T, heads, d], pos [T]: channels i and i + dims / 2 of the first ``dims`` turn by pos * base^(-2i / dims)."""
    out, half = x.clone(), dims // 2
    for i in range(half):
        a = (pos * base ** (-2.0 * i / dims))[:, None]
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., i + half] = v * torch.cos(a) + u * torch.sin(a)
    return out


def windowed_weights(s, window):
    """s [T, T] scores -> weights e^s / (1 + sum e^s) over the ``window`` last columns up to the diagonal."""
    T = s.shape[0]
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    s = s.masked_fill((d < 0) | (d >= window), float("-inf"))
    top = s.max(-1, keepdim=True).values.clamp(min=0)
    e = torch.exp(s - top)
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def attend(q, k, v, scale, window):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv], one head at a time."""
    R = q.shape[1] // k.shape[1]
    return torch.stack([windowed_weights(q[:, h] @ k[:, h // R].T * scale, window) @ v[:, h // R] for h in range(q.shape[1])], dim=1)


def attention(h, W, p, m):
    """Windowed attention with a sink and a gate per head."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    pos = torch.arange(T, dtype=h.dtype)
    q = rotate_halves((h @ W[p + "q"].T).reshape(T, H, -1), pos, m["rot"]["base"], m["rot"]["dims"])
    k = rotate_halves((h @ W[p + "k"].T).reshape(T, G, -1), pos, m["rot"]["base"], m["rot"]["dims"])
    o = attend(q, k, (h @ W[p + "v"].T).reshape(T, G, -1), m["scale"], m["mask"]["size"])
    return (o * sigmoid(h @ W[p + "g"].T)[:, :, None]).reshape(T, -1) @ W[p + "o"].T


def normed_attention(h, W, p, m, eps):
    """The same with biases, norms of the whole query and key rows and of every value head, and no gate."""
    T, H, G = h.shape[0], m["heads"], m["kv_heads"]
    pos = torch.arange(T, dtype=h.dtype)
    row = lambda n: h @ W[p + n].T + W[p + n + ".b"]
    q = (rms_unit(row("q"), eps) * W[p + "q.norm"]).reshape(T, H, -1)
    k = (rms_unit(row("k"), eps) * W[p + "k.norm"]).reshape(T, G, -1)
    v = rms_unit(row("v").reshape(T, G, -1), eps)
    q, k = (rotate_halves(x, pos, m["rot"]["base"], m["rot"]["dims"]) for x in (q, k))
    return attend(q, k, v, m["scale"], m["mask"]["size"]).reshape(T, -1) @ W[p + "o"].T


def causal_conv(u, w):
    """u [T, C], w [C, K]: out[t] = sum_k w[:, k] u[t - (K - 1) + k], zeros before the start."""
    T, K = u.shape[0], w.shape[1]
    out = torch.zeros_like(u)
    for t in range(T):
        for k in range(K):
            s = t - (K - 1) + k
            if s >= 0:
                out[t] += w[:, k] * u[s]
    return out


def gated_delta(q, k, v, g, beta):
    """q, k [T, H, d], v [T, H, dv], g, beta [T, H]: S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=q.dtype)
    out = []
    for t in range(q.shape[0]):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hcv,hc->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hcv,hc->hv", S, q[t]))
    return torch.stack(out)


def delta_mixer(h, W, p, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ W[p + n].T, W[p + n + ".conv"])) for n in "qkv")
    q = unit(q.reshape(T, G, d)).repeat_interleave(H // G, 1) * d ** -0.5
    k = unit(k.reshape(T, G, d)).repeat_interleave(H // G, 1)
    g = torch.exp(-torch.exp(W[p + "A_log"]) * softplus(h @ W[p + "a"].T + W[p + "dt_bias"]))
    o = gated_delta(q, k, v.reshape(T, H, dv), g, sigmoid(h @ W[p + "b"].T))
    o = rms_unit(o, eps) * W[p + "norm"] * silu(h @ W[p + "g"].T).reshape(T, H, dv)
    return o.reshape(T, -1) @ W[p + "o"].T


def channel_delta(r, k, v, w, a):
    """all [T, H, d]: with u = unit(k), S <- diag(w) S - (a u) (u^T S) + k v^T (both terms read the old S); o = S^T r."""
    T, H, d = r.shape
    S = torch.zeros(H, d, d, dtype=r.dtype)
    u = unit(k)
    out = []
    for t in range(T):
        seen = torch.einsum("hcv,hc->hv", S, u[t])
        S = w[t][:, :, None] * S - (a[t] * u[t])[:, :, None] * seen[:, None, :] + k[t][:, :, None] * v[t][:, None, :]
        out.append(torch.einsum("hcv,hc->hv", S, r[t]))
    return torch.stack(out)


def channel_delta_mixer(h, W, p, m, eps):
    heads = lambda x: x.reshape(h.shape[0], m["heads"], m["dim"])
    row = lambda n: h @ W[p + n].T
    w = torch.exp(-math.exp(-0.5) * sigmoid(torch.tanh(row("w1")) @ W[p + "w2"].T + W[p + "w0"]))
    a = sigmoid(row("a") + W[p + "a.b"])
    o = channel_delta(heads(row("r")), heads(row("k")), heads(row("v")), heads(w), heads(a))
    o = rms_unit(o, eps).reshape(h.shape[0], -1) * W[p + "norm"] * sigmoid(row("g"))
    return o @ W[p + "o"].T


def parallel_mixer(h, W, p, m, eps):
    return m["left_scale"] * normed_attention(h, W, p + "left.", m["left"], eps) \
        + m["right_scale"] * channel_delta_mixer(h, W, p + "right.", m["right"], eps)


def dense(h, W, p):
    return xielu(h @ W[p + "up"].T, *W[p + "act"]) @ W[p + "down"].T


def forward(cfg, weights, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one sequence.  ``trace``: a list that receives the stream after every layer."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{layer.get('weights_of', i)}.", layer["mixer"]
        h = rms_unit(x, eps) * W[p + "norm1"]
        if layer["type"] == "attention":
            y = attention(h, W, p + "mix.", m)
        elif layer["type"] == "parallel":
            y = parallel_mixer(h, W, p + "mix.", m, eps)
        else:
            y = delta_mixer(h, W, p + "mix.", m, eps)
        x = x + y
        if layer.get("mlp") is not None:
            x = x + dense(rms_unit(x, eps) * W[p + "norm2"], W, p + "mlp.")
        if trace is not None:
            trace.append(x.clone())
    z = (rms_unit(x, eps) * W["final.norm"]) @ W["head"].T
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(z / cap) if cap else z
