"""A plain, slow implementation of the Viperax design: one function per mechanism, whole sequences, no cache, no batching, float64
arithmetic on the CPU. It shares no code with the engine; the tests hold the engine to it.

A model is (config dict, {tensor name: torch tensor}); weights are widened exactly. Notation: X [S, T, W] are the S residual streams of one
sequence whose tokens stand at positions 0..T-1; W_foo y means y @ W_foo.T.

`rnd` (None or torch.bfloat16) rounds where an engine that serves in that precision may round: the inputs of the matrix products (normed
activations, queries, the cached latents, queries in the latent space, attention results, the gated heads, hidden activations). What the
design wants in 32-bit stays unrounded. The difference between the two is the size of the rounding noise that the tests measure the
bfloat16 engine by.
"""
from __future__ import annotations

import torch

F = torch.float64


def w(tensors, name):
    return tensors[name].to(F)


def rounded(x, rnd):
    return x if rnd is None else x.to(rnd).to(F)


def layer_norm(x, gain, eps):
    """(x - mean) / sqrt(mean((x - mean)^2) + eps) * gain along the last axis."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * gain


def rms_norm(x, gain, eps):
    """x / sqrt(mean(x^2) + eps) * gain along the last axis."""
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps) * gain


def silu(z):
    return z * torch.sigmoid(z)


def embed(tensors, cfg, tokens):
    """[T, W]: the tokens' rows of the table, scaled."""
    return w(tensors, "embed")[torch.as_tensor(tokens)] * cfg["embedding"]["scale"]


def read_streams(X, weights):
    """u = sum_s weights[s] X_s."""
    u = torch.zeros_like(X[0])
    for s in range(X.shape[0]):
        u = u + weights[s] * X[s]
    return u


def write_streams(X, mix, out, y):
    """X'_t = sum_s mix[s, t] X_s + out[t] y, every X' from the old X."""
    new = []
    for t in range(X.shape[0]):
        v = out[t] * y
        for s in range(X.shape[0]):
            v = v + mix[s, t] * X[s]
        new.append(v)
    return torch.stack(new)


def visible(T, window):
    """[T, T] bool: i sees j if 0 <= i - j < window (window 0: every earlier key)."""
    i, j = torch.arange(T).view(-1, 1), torch.arange(T).view(1, -1)
    d = i - j
    return (d >= 0) & (d < window) if window else d >= 0


def sink_softmax(scores, seen, sink):
    """exp(score) / (sum over the seen keys of exp(score) + exp(sink)) per row; scores [T, T], sink a number."""
    s = torch.where(seen, scores, torch.full_like(scores, -torch.inf))
    m = torch.maximum(s.max(-1, keepdim=True).values, sink.view(1, 1))
    e = torch.exp(s - m)
    return e / (e.sum(-1, keepdim=True) + torch.exp(sink - m))


def latents(h, tensors, p, eps, rnd=None):
    """c [T, R]: the normed key/value latent of every token, as a cache holds it."""
    c = rms_norm(h @ w(tensors, p + "dkv").T, w(tensors, p + "dkv.norm"), eps)
    return rounded(c, rnd)


def latent_attention(h, c, tensors, p, m, rnd=None):
    """h [T, W] the mixer's input, c [T, R] the latents (this layer's own or another layer's); returns the mixer's result [T, W]."""
    T, H, D, V = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = rounded(h @ w(tensors, p + "q").T, rnd).view(T, H, D)
    gate = torch.sigmoid(h @ w(tensors, p + "g").T)
    uk, uv = w(tensors, p + "uk").view(H, D, -1), w(tensors, p + "uv").view(H, V, -1)
    seen = visible(T, (m.get("mask") or {}).get("size", 0))
    heads = []
    for a in range(H):
        if rnd is None:
            scores = (q[:, a] @ (c @ uk[a].T).T) * m["scale"]
            heads.append(sink_softmax(scores, seen, w(tensors, p + "sink")[a]) @ (c @ uv[a].T))
        else:       # the key projection taken into the query: q.(U c) = (U^T q).c, and the value projection behind the weights' sum
            scores = (rounded(q[:, a] @ uk[a], rnd) @ c.T) * m["scale"]
            heads.append(rounded(sink_softmax(scores, seen, w(tensors, p + "sink")[a]) @ c, rnd) @ uv[a].T)
    y = rounded(torch.cat(heads, dim=1) * gate, rnd)
    return y @ w(tensors, p + "o").T


def gated(h, tensors, p, rnd=None):
    """W_down (silu(W_gate h) * (W_up h))."""
    z = silu(h @ w(tensors, p + "gate").T) * (h @ w(tensors, p + "up").T)
    return rounded(z, rnd) @ w(tensors, p + "down").T


def table_experts(h, tokens, tensors, p, mlp, rnd=None):
    """The experts that a stored table gives each token id, every one with weight 1 / top, and the shared expert."""
    table, top = tensors[p + "table"], mlp["router"]["top"]
    y = torch.zeros_like(h)
    for i, t in enumerate(tokens):
        for k in range(top):
            y[i] = y[i] + gated(h[i:i + 1], tensors, f"{p}e{int(table[t, k])}.", rnd)[0] / top
    if mlp.get("shared"):
        y = y + gated(h, tensors, p + "shared.", rnd)
    return y


def feed_forward(h, tokens, tensors, p, mlp, rnd=None):
    return gated(h, tensors, p, rnd) if mlp["kind"] == "dense" else table_experts(h, tokens, tensors, p, mlp, rnd)


def run(cfg, tensors, tokens, rnd=None, after_layer=None):
    """Logits [T, vocab] of a whole sequence; `after_layer(i, x)` sees the sum of the streams behind every layer."""
    eps = cfg["norm"]["eps"]
    e = embed(tensors, cfg, tokens)
    X = torch.stack([e] * cfg["streams"])
    cached = {}
    for i, layer in enumerate(cfg["layers"]):
        p, m = f"l{i}.", layer["mixer"]
        h = rounded(layer_norm(read_streams(X, w(tensors, p + "hc1.in")), w(tensors, p + "norm1"), eps), rnd)
        if m.get("kv_from") is None:
            cached[i] = latents(h, tensors, p + "mix.", eps, rnd)
        c = cached[i if m.get("kv_from") is None else m["kv_from"]]
        y = latent_attention(h, c, tensors, p + "mix.", m, rnd)
        X = write_streams(X, w(tensors, p + "hc1.mix"), w(tensors, p + "hc1.out"), y)
        if layer.get("mlp"):
            h = rounded(layer_norm(read_streams(X, w(tensors, p + "hc2.in")), w(tensors, p + "norm2"), eps), rnd)
            y = feed_forward(h, tokens, tensors, p + "mlp.", layer["mlp"], rnd)
            X = write_streams(X, w(tensors, p + "hc2.mix"), w(tensors, p + "hc2.out"), y)
        if after_layer is not None:
            after_layer(i, X.sum(0))
    return head(layer_norm(X.sum(0), w(tensors, "final.norm"), eps), cfg, tensors, rnd)


def head(x, cfg, tensors, rnd=None):
    """logits = W x * logit_scale, then cap * tanh(logits / cap)."""
    logits = (rounded(x, rnd) @ w(tensors, "head").T) * cfg.get("logit_scale", 1.0)
    cap = cfg.get("logit_softcap")
    return cap * torch.tanh(logits / cap) if cap else logits
