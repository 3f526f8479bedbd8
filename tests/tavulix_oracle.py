"""Slow, plain restatement of the Tavulix decoder for the tests: one function per mechanism, whole
sequences at once, no cache, no batching, nothing imported from the package under test.

Notation: T tokens, D channels of the residual stream; all arithmetic in the dtype of the weights
handed in (float64 in most tests)."""
import torch


def rms_unit(x, eps):
    """u = x / sqrt(<x^2> + eps) along the last axis."""
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def causal_conv(u, w):
    """u [T, C], w [C, K]: out[t, c] = sum_k w[c, k] u[t - (K - 1) + k, c], with u[<0] = 0."""
    T, C = u.shape
    K = w.shape[1]
    out = torch.zeros_like(u)
    for t in range(T):
        for k in range(K):
            s = t - (K - 1) + k
            if s >= 0:
                out[t] += w[:, k] * u[s]
    return out


def soft_cap(s, cap):
    return s if cap is None else cap * torch.tanh(s / cap)


def log_distance(r1, r2, dist):
    """Penalty of one head at the given distances (a tensor >= 0)."""
    return r1 * torch.log(1.0 + r2 * dist)


def visible(i, j, size, keep):
    """Does position i attend to position j?"""
    if j > i:
        return False
    return size is None or i - j < size or j < keep


def visibility(T, size, keep):
    i = torch.arange(T)[:, None]
    j = torch.arange(T)[None, :]
    near = torch.ones(T, T, dtype=torch.bool) if size is None else (i - j < size)
    return (j <= i) & (near | (j < keep))


def sink_softmax(scores, mask, sink):
    """scores [T, S], mask bool [T, S], sink: number or None.  Rows sum to less than 1 with a sink."""
    s = scores.masked_fill(~mask, float("-inf"))
    top = s.max(dim=-1, keepdim=True).values
    if sink is not None:
        top = torch.maximum(top, sink.reshape(1, 1).expand_as(top))
    e = torch.exp(s - top)
    den = e.sum(-1, keepdim=True)
    if sink is not None:
        den = den + torch.exp(sink - top)
    return e / den


def attend(q, k, v, *, scale, cap, r1, r2, sink, size, keep):
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv], one head at a time."""
    T, H, _ = q.shape
    G = k.shape[1]
    pos = torch.arange(T, dtype=q.dtype)
    dist = (pos[:, None] - pos[None, :]).clamp_min(0)
    mask = visibility(T, size, keep)
    outs = []
    for h in range(H):
        g = h // (H // G)
        s = soft_cap((q[:, h] @ k[:, g].T) * scale, cap)
        if r1 is not None:
            s = s - log_distance(r1[h], r2[h], dist)
        outs.append(sink_softmax(s, mask, None if sink is None else sink[h]) @ v[:, g])
    return torch.stack(outs, dim=1)


def mix_values(v, v_first, lam):
    return (1 - lam) * v + lam * v_first


def poly_norm(z, coef, eps):
    a, b, c, e = coef[0], coef[1], coef[2], coef[3]
    return a * rms_unit(z, eps) + b * rms_unit(z * z, eps) + c * rms_unit(z * z * z, eps) + e


def attention_mixer(h, W, p, m, eps, v_first):
    """h [T, D]; W: tensors by name, p: prefix of the layer's mixer, m: its config entry.
    Returns (output [T, D], the layer's values before mixing)."""
    T = h.shape[0]
    H, G, d, dv = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    proj = {}
    for n in "qkv":
        u = h @ W[p + n].T
        cw = W.get(p + n + ".conv")
        proj[n] = u if cw is None else causal_conv(u, cw)
    q = rms_unit(proj["q"].reshape(T, H, d), eps) * W[p + "q.norm"]
    k = rms_unit(proj["k"].reshape(T, G, d), eps) * W[p + "k.norm"]
    own = proj["v"].reshape(T, G, dv)
    v = own
    if m.get("v_mix") and v_first is not None:
        v = mix_values(own, v_first, W[p + "vmix"])
    mask = m.get("mask") or {}
    o = attend(q, k, v, scale=m["scale"], cap=m.get("softcap"), r1=W.get(p + "r1"), r2=W.get(p + "r2"),
               sink=W.get(p + "sink"), size=mask.get("size"), keep=mask.get("keep_first", 0))
    gate = torch.sigmoid(h @ W[p + "g"].T)
    o = o * gate[:, :, None]
    return o.reshape(T, H * dv) @ W[p + "o"].T, own


def forward(cfg, weights, tokens, dtype=torch.float64, trace=None):
    """Logits [T, vocab] of one sequence.  ``trace``: a list that receives the stream after every layer."""
    W = {n: t.to(dtype) for n, t in weights.items()}
    ids = torch.as_tensor(tokens, dtype=torch.long)
    eps = cfg["norm"]["eps"]
    x = W["embed"][ids] + W["pos"][: len(ids)]
    v_first = None
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        y, own = attention_mixer(rms_unit(x, eps) * W[p + "norm1"], W, p + "mix.", layer["mixer"], eps, v_first)
        if layer["mixer"].get("v_mix") and v_first is None:
            v_first = own
        x = x + rms_unit(y, eps) * W[p + "norm1b"]
        if layer.get("mlp") is not None:
            z = (rms_unit(x, eps) * W[p + "norm2"]) @ W[p + "mlp.up"].T
            y = poly_norm(z, W[p + "mlp.act"], eps) @ W[p + "mlp.down"].T
            x = x + rms_unit(y, eps) * W[p + "norm2b"]
        if trace is not None:
            trace.append(x.clone())
    return soft_cap((rms_unit(x, eps) * W["final.norm"]) @ W["head"].T, cfg.get("logit_softcap"))
