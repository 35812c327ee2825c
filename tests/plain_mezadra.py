"""A plain, slow implementation of the Mezadra design: one function per mechanism, whole sequences, no cache, no batching, float64
arithmetic on the CPU. It shares no code with the engine; the tests hold the engine to it.

A model is (config dict, {tensor name: torch tensor}); weights are widened exactly. Notation: x [T, W] is the residual of one sequence whose
tokens stand at positions 0..T-1; W_foo y means y @ W_foo.T.

`rnd` (None or torch.bfloat16) rounds where an engine that serves in that precision may round: the inputs of the matrix products (the
residual as a sublayer reads it, normed queries and keys, the cached keys and values, attention results, gated heads, hidden activations).
What the design wants in 32-bit stays unrounded. The difference between the two is the size of the rounding noise that the tests measure the
bfloat16 engine by.
"""
from __future__ import annotations

import torch

F = torch.float64


def w(tensors, name):
    return tensors[name].to(F)


def rounded(x, rnd):
    return x if rnd is None else x.to(rnd).to(F)


def unit_rms(x, eps):
    """x / sqrt(mean(x^2) + eps) along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def embed(tensors, cfg, tokens):
    """[T, W]: the tokens' rows of the table, scaled."""
    return w(tensors, "embed")[torch.as_tensor(tokens)] * cfg.get("embedding", {}).get("scale", 1.0)


def short_conv(u, taps):
    """y_t[c] = sum_j taps[c, j] u_(t - K + 1 + j)[c], zeros before the start; u [T, C], taps [C, K]."""
    T, K = u.shape[0], taps.shape[1]
    y = torch.zeros_like(u)
    for t in range(T):
        for j in range(K):
            at = t - K + 1 + j
            if at >= 0:
                y[t] += taps[:, j] * u[at]
    return y


def rotated(x, base, dims, first=0):
    """x [T, heads, D] at positions first ..: elements i and i + dims / 2 of a head, i < dims / 2, turned by position * base^(-2i / dims)."""
    half = dims // 2
    a = torch.arange(first, first + x.shape[0], dtype=F).view(-1, 1) * base ** (-2.0 * torch.arange(half, dtype=F) / dims)
    c, s = torch.cos(a).unsqueeze(1), torch.sin(a).unsqueeze(1)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def capped(scores, cap):
    return cap * torch.tanh(scores / cap) if cap else scores


def sink_softmax(scores, sink):
    """exp(score) / (sum over j <= i of exp(score) + exp(sink)) per row; scores [T, T], sink a number."""
    T = scores.shape[0]
    s = torch.where(torch.ones(T, T).tril().bool(), scores, torch.full_like(scores, -torch.inf))
    m = torch.maximum(s.max(-1, keepdim=True).values, sink.view(1, 1))
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def attention(h, tensors, p, m, eps, first_values=None, rnd=None):
    """h [T, W] the mixer's input; `first_values` [T, G Dv] or None: what the values are mixed with. Returns (result [T, W], the layer's own
    values in front of the mixing [T, G Dv])."""
    T, H, G, D, V = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (h @ w(tensors, p + r).T for r in "qkv")
    if m.get("conv"):
        q, k, v = (short_conv(u, w(tensors, p + r + ".conv")) for u, r in ((q, "q"), (k, "k"), (v, "v")))
    own = v
    if first_values is not None:
        lam = w(tensors, p + "vmix")
        v = (1.0 - lam) * v + lam * first_values
    q, k, v = q.view(T, H, D), k.view(T, G, D), rounded(v, rnd).view(T, G, V)
    if m.get("rot"):
        q, k = (rotated(y, m["rot"]["base"], m["rot"]["dims"]) for y in (q, k))
    q, k = rounded(unit_rms(q, eps), rnd), rounded(unit_rms(k, eps), rnd)
    heads = []
    for a in range(H):
        g = a // (H // G)
        scores = capped((q[:, a] @ k[:, g].T) * m["scale"], m.get("softcap"))
        heads.append(sink_softmax(scores, w(tensors, p + "sink")[a]) @ v[:, g])
    return rounded(torch.cat(heads, dim=1), rnd) @ w(tensors, p + "o").T, own


def linear_recurrence(q, k, v, decay):
    """S_t = decay_h S_(t-1) + k_t v_t^T, o_t = S_t^T q_t per head; q, k [T, H, D], v [T, H, V], decay [H]; o [T, H, V]."""
    S = torch.zeros(q.shape[1], q.shape[2], v.shape[2], dtype=F)
    out = []
    for t in range(q.shape[0]):
        S = decay.view(-1, 1, 1) * S + k[t].unsqueeze(2) * v[t].unsqueeze(1)
        out.append((S * q[t].unsqueeze(2)).sum(1))
    return torch.stack(out)


def lightning(h, tensors, p, m, eps, rnd=None):
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (silu(h @ w(tensors, p + r).T) for r in "qkv")
    o = linear_recurrence(q.view(T, H, D), k.view(T, H, D), v.view(T, H, V), torch.tensor(m["decay"], dtype=F)).reshape(T, H * V)
    y = unit_rms(o, eps) * w(tensors, p + "norm") * torch.sigmoid(h @ w(tensors, p + "g").T)
    return rounded(y, rnd) @ w(tensors, p + "o").T


def clamped_gated(h, tensors, p, limit, rnd=None):
    """g = min(W_gate h, limit), u = W_up h clamped to +-limit; W_down (g sigmoid(1.702 g) (u + 1))."""
    g, u = torch.clamp(h @ w(tensors, p + "gate").T, max=limit), torch.clamp(h @ w(tensors, p + "up").T, -limit, limit)
    return rounded(g * torch.sigmoid(1.702 * g) * (u + 1.0), rnd) @ w(tensors, p + "down").T


def gated(h, tensors, p, rnd=None):
    """W_down (silu(W_gate h) * (W_up h))."""
    return rounded(silu(h @ w(tensors, p + "gate").T) * (h @ w(tensors, p + "up").T), rnd) @ w(tensors, p + "down").T


def route(h, tensors, p, top):
    """Per token: [(expert, weight)], the `top` largest sigmoids of the router's logits, as they are."""
    s = torch.sigmoid(h @ w(tensors, p + "router").T)
    return [[(int(e), s[t, e]) for e in torch.topk(s[t], top).indices] for t in range(h.shape[0])]


def experts(h, tensors, p, mlp, rnd=None):
    """The sum of expert(weight * h) over a token's experts, and the shared expert times sigmoid(W_sg h)."""
    y = torch.zeros_like(h)
    for t, chosen in enumerate(route(h, tensors, p, mlp["router"]["top"])):
        for e, weight in chosen:
            y[t] += gated(weight * h[t:t + 1], tensors, f"{p}e{e}.", rnd)[0]
    if mlp.get("shared"):
        y = y + gated(h, tensors, p + "shared.", rnd) * torch.sigmoid(h @ w(tensors, p + "shared.sg").T)
    return y


def feed_forward(h, tensors, p, mlp, rnd=None):
    return clamped_gated(h, tensors, p, mlp["limit"], rnd) if mlp["kind"] == "dense" else experts(h, tensors, p, mlp, rnd)


def run(cfg, tensors, tokens, rnd=None, after_layer=None):
    """Logits [T, vocab] of a whole sequence; `after_layer(i, x)` sees the residual behind every layer."""
    eps = cfg["norm"]["eps"]
    x = embed(tensors, cfg, tokens)
    first_values = None
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rounded(x, rnd)
        if layer["type"] == "attention":
            mixes = bool(m.get("v_mix"))
            y, own = attention(h, tensors, p + "mix.", m, eps, first_values if mixes else None, rnd)
            if mixes and first_values is None:
                first_values = own
        else:
            y = lightning(h, tensors, p + "mix.", m, eps, rnd)
        x = x + unit_rms(y, eps) * w(tensors, p + "norm1")
        if layer.get("mlp"):
            x = x + unit_rms(feed_forward(rounded(x, rnd), tensors, p + "mlp.", layer["mlp"], rnd), eps) * w(tensors, p + "norm2")
        if after_layer is not None:
            after_layer(i, x)
    return rounded(unit_rms(x, eps) * w(tensors, "final.norm"), rnd) @ w(tensors, "head").T
