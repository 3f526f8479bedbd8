"""Slow, plain restatement of the Milivik decoder for the tests: one function per mechanism, whole sequences at once,
no cache, no batching, nothing imported from the package under test.

Notation: T tokens, D channels of the residual stream, `<.>` a mean over the last axis; arithmetic in the dtype of the
weights handed in (float64 in most tests)."""
import math

import torch


def unit(x, eps):
    """x / sqrt(<x^2> + eps)."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def branch_norm(y, w, eps):
    """Norm of a branch before it joins the stream; the gain is stored less one."""
    return unit(y, eps) * (1 + w)


def silu(z):
    return z / (1 + torch.exp(-z))


def sigmoid(z):
    return 1 / (1 + torch.exp(-z))


# ------------------------------------------------------------------------------------------ rotation
def yarn_frequencies(dims, base, scaling):
    """(frequency of every pair [dims / 2], factor on cos and sin).  Pairs that turn more than `fast` times over the original
    length keep their frequency, those below `slow` turns are slowed by `factor`, a ramp lies between."""
    f = [base ** (-2.0 * i / dims) for i in range(dims // 2)]
    if scaling is None:
        return torch.tensor(f, dtype=torch.float64), 1.0
    pair_at = lambda turns: dims * math.log(scaling["original"] / (2 * math.pi * turns)) / (2 * math.log(base))
    lo = max(math.floor(pair_at(scaling["fast"])), 0)
    hi = min(math.ceil(pair_at(scaling["slow"])), dims - 1)
    out = []
    for i, fi in enumerate(f):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(fi / scaling["factor"] * r + fi * (1 - r))
    return torch.tensor(out, dtype=torch.float64), 0.1 * math.log(scaling["factor"]) + 1


def rotate_halves(x, pos, freq, mag=1.0):
    """x [T, ..., n], pos [T]: channels (i, i + n / 2) turn by pos * freq[i] and grow by mag."""
    half = x.shape[-1] // 2
    out = x.clone()
    for i in range(half):
        a = (pos.double() * freq[i]).reshape(-1, *([1] * (x.dim() - 2)))
        c, s = (mag * torch.cos(a)).to(x.dtype), (mag * torch.sin(a)).to(x.dtype)
        u, v = x[..., i], x[..., i + half]
        out[..., i] = u * c - v * s
        out[..., i + half] = v * c + u * s
    return out


# ------------------------------------------------------------------------------------------ attention
def visible(T, size=None):
    """[T, T]: row i sees columns j <= i, with a window only the last `size` of them."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    see = j <= i
    return see if size is None else see & (i - j < size)


def masked_softmax(s, see):
    s = s.masked_fill(~see, float("-inf"))
    e = torch.exp(s - s.max(-1, keepdim=True).values)
    return e / e.sum(-1, keepdim=True)


def attend_latent(q_u, q_r, c, kr, uk, uv, scale, size=None):
    """q_u [T, H, d], q_r [T, H, r] (rotated), c [T, rank], kr [T, r] (rotated), uk [H, d, rank], uv [H, dv, rank]
    -> [T, H, dv], one head at a time."""
    see, outs = visible(q_u.shape[0], size), []
    for n in range(q_u.shape[1]):
        s = (q_u[:, n] @ (c @ uk[n].T).T + q_r[:, n] @ kr.T) * scale
        outs.append(masked_softmax(s, see) @ (c @ uv[n].T))
    return torch.stack(outs, dim=1)


def latent_mixer(h, W, p, m, eps):
    T, H, d, r, dv, rank = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    freq, mag = yarn_frequencies(r, m["rot"]["base"], m["rot"].get("scaling"))
    q = (unit(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]) @ W[p + "uq"].T
    q = q.reshape(T, H, d + r)
    z = h @ W[p + "dkv"].T
    c = unit(z[:, :rank], eps) * W[p + "dkv.norm"]
    size = (m.get("mask") or {}).get("size")
    o = attend_latent(q[:, :, :d], rotate_halves(q[:, :, d:], pos, freq, mag), c, rotate_halves(z[:, rank:], pos, freq, mag),
                      W[p + "uk"].reshape(H, d, rank), W[p + "uv"].reshape(H, dv, rank), m["scale"], size)
    return (o.reshape(T, H * dv) * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def query_temperature(pos, coef, every):
    """Factor on the queries of a position: 1 + coef ln(1 + how many whole periods the position has completed)."""
    return torch.tensor([1 + coef * math.log((int(p) + 1) // every + 1) for p in pos], dtype=torch.float64)


def attend_maps(q, k, v, scale, see=None):
    """q [T, H, 2, d], k [T, G, 2, d], v [T, G, dv] -> the results of both maps [T, H, 2, dv]."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    see = visible(T) if see is None else see
    out = torch.empty(T, H, 2, v.shape[2], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        for m in range(2):
            out[:, h, m] = masked_softmax(q[:, h, m] @ k[:, g, m].T * scale, see) @ v[:, g]
    return out


def diff_lambda(lq1, lk1, lq2, lk2, diff):
    return math.exp(float((lq1 * lk1).sum())) - math.exp(float((lq2 * lk2).sum())) + diff


def combine_maps(a, lam, diff, eps):
    """a [T, H, 2, dv] -> [T, H, dv]: first map less lam times the second, normed per head, times 1 - diff."""
    return unit(a[:, :, 0] - lam * a[:, :, 1], eps) * (1 - diff)


def diff_mixer(h, W, p, m, eps):
    T, H, G, d, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = unit((h @ W[p + "q"].T).reshape(T, H, 2, d), eps) * W[p + "q.norm"]
    k = unit((h @ W[p + "k"].T).reshape(T, G, 2, d), eps) * W[p + "k.norm"]
    v = (h @ W[p + "v"].T).reshape(T, G, dv)
    if m.get("q_temp"):
        q = q * query_temperature(range(T), m["q_temp"]["coef"], m["q_temp"]["every"]).to(q.dtype)[:, None, None, None]
    lam = diff_lambda(*(W[p + n] for n in ("lq1", "lk1", "lq2", "lk2")), m["diff"])
    o = combine_maps(attend_maps(q, k, v, m["scale"]), lam, m["diff"], eps)
    return (o * sigmoid(h @ W[p + "g"].T)[:, :, None]).reshape(T, H * dv) @ W[p + "o"].T


# --------------------------------------------------------------------------------------- feed-forward
def gated_ff(h, W, p):
    return (silu(h @ W[p + "gate"].T) * (h @ W[p + "up"].T)) @ W[p + "down"].T


def route(z, top, count=None, keep=None, scale=1.0):
    """z [E] of one token -> (ids, weights).  Scores are sigmoids; of `count` groups of neighbours the `keep` best (by the
    sum of their two best scores) take part."""
    s = [1 / (1 + math.exp(-float(v))) for v in z]
    live = list(range(len(s)))
    if count is not None:
        n = len(s) // count
        groups = [live[g * n:(g + 1) * n] for g in range(count)]
        best = sorted(groups, key=lambda g: -sum(sorted((s[e] for e in g), reverse=True)[:2]))[:keep]
        live = [e for g in best for e in g]
    ids = sorted(live, key=lambda e: -s[e])[:top]
    total = sum(s[e] for e in ids) + 1e-20
    return ids, [s[e] / total * scale for e in ids]


def steady(z, spread, *rule):
    """Does the choice of one token stay the same when its logits move by about ``spread``?"""
    g = torch.Generator().manual_seed(0)
    ids = set(route(z, *rule)[0])
    return all(set(route(z + spread * torch.randn(z.shape, generator=g, dtype=z.dtype), *rule)[0]) == ids for _ in range(8))


def mixture(h, W, p, m, clear=None):
    r = m["router"]
    g = r.get("groups") or {}
    z = h @ W[p + "router"].T
    weight = torch.zeros_like(z)
    for t in range(h.shape[0]):
        rule = r["top"], g.get("count"), g.get("keep"), r["scale"]
        for e, w in zip(*route(z[t], *rule)):
            weight[t, e] = w
        if clear is not None:
            clear[t] &= steady(z[t], 0.03, *rule)
    out = sum(weight[:, e:e + 1] * gated_ff(h, W, f"{p}e{e}.") for e in range(r["experts"]))
    if m.get("shared"):
        out = out + sigmoid(h @ W[p + "shared.sg"].T) * gated_ff(h, W, p + "shared.")
    return out


# ---------------------------------------------------------------------------------------------- model
def forward(cfg, weights, tokens, dtype=torch.float64, trace=None, clear=None):
    """Logits [T, vocab] of one sequence.  ``trace``: a list that receives the stream after every layer; ``clear`` (bool
    [T]): cleared where a router's choice is so close that rounding to bf16 may turn it."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    ids = torch.as_tensor(tokens, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    x = W["embed"][ids] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p, mix = f"l{i}.", {"latent_attention": latent_mixer, "attention": diff_mixer}[layer["type"]]
        x = x + branch_norm(mix(x, W, p + "mix.", layer["mixer"], eps), W[p + "norm1"], eps)
        m = layer.get("mlp")
        if m is not None:
            y = gated_ff(x, W, p + "mlp.") if m["kind"] == "dense" else mixture(x, W, p + "mlp.", m, clear)
            x = x + branch_norm(y, W[p + "norm2"], eps)
        if trace is not None:
            trace.append(x.clone())
    return branch_norm(x, W["final.norm"], eps) @ W["embed"].T * cfg["logit_scale"]
