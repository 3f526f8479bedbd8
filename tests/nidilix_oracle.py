"""Slow, plain restatement of the Nidilix decoder for the tests: one function per mechanism, whole sequences
at once, no cache, no batching, nothing imported from the package under test.

Notation: T tokens, D channels of the residual stream, `<.>` a mean over the last axis; arithmetic in the dtype
of the weights handed in (float64 in most tests)."""
import math

import torch


def rms_unit(x, eps):
    """x / sqrt(<x^2> + eps)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def tanh_norm(x, alpha, w, b):
    """A norm without statistics: w tanh(alpha x) + b."""
    return w * torch.tanh(alpha * x) + b


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def relu_squared(z):
    r = torch.clamp(z, min=0)
    return r * r


def rotate_pairs(x, pos, base):
    """x [T, ..., n], pos [T]: channels (2i, 2i + 1) turn by pos * base^(-2i / n)."""
    n = x.shape[-1]
    out = x.clone()
    for i in range(n // 2):
        a = pos * base ** (-2.0 * i / n)
        a = a.reshape(-1, *([1] * (x.dim() - 2)))
        u, v = x[..., 2 * i], x[..., 2 * i + 1]
        out[..., 2 * i] = u * torch.cos(a) - v * torch.sin(a)
        out[..., 2 * i + 1] = v * torch.cos(a) + u * torch.sin(a)
    return out


def latent_of(h, w_dkv, norm_w, rank, base, eps):
    """What a token leaves in the cache: (normed latent [T, rank], rotated key part shared by the heads)."""
    z = h @ w_dkv.T
    pos = torch.arange(h.shape[0], dtype=h.dtype)
    return rms_unit(z[:, :rank], eps) * norm_w, rotate_pairs(z[:, rank:], pos, base)


def causal_softmax(s):
    """s [T, T] -> weights of row i over columns j <= i."""
    T = s.shape[0]
    future = torch.arange(T)[None, :] > torch.arange(T)[:, None]
    s = s.masked_fill(future, float("-inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def attend_latent(q_u, q_r, c, kr, uk, uv, scale):
    """q_u [T, H, d], q_r [T, H, r] (rotated), c [T, rank], kr [T, r] (rotated), uk [H, d, rank], uv [H, dv, rank]
    -> [T, H, dv], one head at a time."""
    outs = []
    for n in range(q_u.shape[1]):
        s = (q_u[:, n] @ (c @ uk[n].T).T + q_r[:, n] @ kr.T) * scale
        outs.append(causal_softmax(s) @ (c @ uv[n].T))
    return torch.stack(outs, dim=1)


def latent_attention(h, latent, W, p, m):
    """h [T, D]; latent: pair from ``latent_of`` (the layer's own or another layer's); m: the mixer's entry."""
    c, kr = latent
    T, H, d, r, dv = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"]
    pos = torch.arange(T, dtype=h.dtype)
    q = (h @ W[p + "q"].T).reshape(T, H, d + r)
    q_r = rotate_pairs(q[:, :, d:], pos, m["rot"]["base"])
    o = attend_latent(q[:, :, :d], q_r, c, kr, W[p + "uk"].reshape(H, d, -1), W[p + "uv"].reshape(H, dv, -1), m["scale"])
    gate = torch.sigmoid(h @ W[p + "g"].T)
    return (o * gate[:, :, None]).reshape(T, H * dv) @ W[p + "o"].T


def causal_conv(u, w, b):
    """u [T, C], w [C, K]: out[t] = b + sum_k w[:, k] u[t - (K - 1) + k], zeros before the start."""
    T, K = u.shape[0], w.shape[1]
    out = b.expand(T, -1).clone()
    for t in range(T):
        for k in range(K):
            s = t - (K - 1) + k
            if s >= 0:
                out[t] += w[:, k] * u[s]
    return out


def block_linear(u, w, b):
    """u [T, C], w [B, n, n] ([out, in] per part), b [B, n]; C = B n."""
    n = w.shape[1]
    return torch.cat([u[:, i * n:(i + 1) * n] @ w[i].T + b[i] for i in range(w.shape[0])], dim=1)


def rglru_scan(u, r, i, lam):
    """S_t = a_t S_(t-1) + sqrt(1 - a_t^2) i_t u_t with ln a = -8 r softplus(lam); all states [T, C]."""
    sp = torch.log1p(torch.exp(-lam.abs())) + lam.clamp(min=0)
    S = torch.zeros_like(u[0])
    out = []
    for t in range(u.shape[0]):
        log_a = -8.0 * r[t] * sp
        S = torch.exp(log_a) * S + torch.sqrt(-torch.expm1(2 * log_a)) * i[t] * u[t]
        out.append(S)
    return torch.stack(out)


def rglru_mixer(h, W, p):
    y = gelu_tanh(h @ W[p + "y"].T + W[p + "y.b"])
    u = causal_conv(h @ W[p + "x"].T + W[p + "x.b"], W[p + "conv"], W[p + "conv.b"])
    r = torch.sigmoid(block_linear(u, W[p + "ra"], W[p + "ra.b"]))
    i = torch.sigmoid(block_linear(u, W[p + "ri"], W[p + "ri.b"]))
    return (rglru_scan(u, r, i, W[p + "lam"]) * y) @ W[p + "o"].T


def expert(h, up, down):
    return relu_squared(h @ up.T) @ down.T


def route(logits, top):
    """[T, E] -> (ids [T, top], weights [T, top]): the largest logits, softmax among themselves."""
    val, ids = torch.sort(logits, dim=-1, descending=True, stable=True)
    val, ids = val[:, :top], ids[:, :top]
    e = torch.exp(val - val[:, :1])
    return ids, e / e.sum(-1, keepdim=True)


def mixture(h, W, p, m):
    ids, wt = route(h @ W[p + "router"].T + W[p + "router.b"], m["router"]["top"])
    out = torch.zeros_like(h)
    for e in range(m["router"]["experts"]):
        w_e = (wt * (ids == e)).sum(-1, keepdim=True)                 # 0 where the expert is not chosen
        out += w_e * expert(h, W[f"{p}e{e}.up"], W[f"{p}e{e}.down"])
    if m.get("shared"):
        out = out + expert(h, W[p + "shared.up"], W[p + "shared.down"])
    return out


def token_side(x, rows, W, p, eps):
    """rows [T, dim]: the layer's part of the side table; returns the branch added to the stream."""
    y = (gelu_tanh(x @ W[p + "gate"].T) * rows) @ W[p + "proj"].T
    return rms_unit(y, eps) * W[p + "norm"]


def forward(cfg, weights, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one sequence.  ``trace``: a list that receives the stream after every layer."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    ids = torch.as_tensor(tokens, dtype=torch.long)
    eps, mult = cfg["norm"]["eps"], cfg["residual_mult"]
    norm = lambda x, n: tanh_norm(x, W[n + ".alpha"], W[n], W[n + ".b"])
    side = cfg.get("token_side")
    x = W["embed"][ids]
    latents = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = norm(x, p + "norm1")
        if layer["type"] == "rglru":
            y = rglru_mixer(h, W, p + "mix.")
        else:
            src = m.get("kv_from")
            if src is None:
                src = i
                latents[i] = latent_of(h, W[p + "mix.dkv"], W[p + "mix.dkv.norm"], m["kv_rank"], m["rot"]["base"], eps)
            y = latent_attention(h, latents[src], W, p + "mix.", m)
        x = x + mult * y
        if layer.get("mlp") is not None:
            x = x + mult * mixture(norm(x, p + "norm2"), W, p + "mlp.", layer["mlp"])
        if side:
            n = side["dim"]
            x = x + mult * token_side(x, W["side.embed"][ids][:, i * n:(i + 1) * n], W, p + "side.", eps)
        if trace is not None:
            trace.append(x.clone())
    return norm(x, "final.norm") @ W["head"].T
