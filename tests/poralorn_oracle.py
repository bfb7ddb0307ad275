"""Plain, slow statement of the Poralorn decoder in float64: one function per mechanism, whole sequences, no cache, no
batching, keys and values always expanded.  It is written from the equations and imports nothing of the package, so the
tests compare two independent programs.  ``weights`` maps checkpoint names to tensors, ``cfg`` is the parsed config.json."""
from __future__ import annotations

import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_erf(z):
    return 0.5 * z * (1 + torch.erf(z / math.sqrt(2.0)))


def sigmoid(z):
    return 1.0 / (1.0 + torch.exp(-z))


def latent(h, w_down, w_norm, eps):
    """What one token leaves behind for later tokens: ``[T, width] -> [T, rank]``."""
    return rms(h @ w_down.T, eps) * w_norm


def latent_attention(q, c, w_key, w_value, scale, start=0):
    """``q [Tq, heads, dim]`` at positions ``start ..`` over latents ``c [T, rank]``; ``w_key [heads * dim, rank]``,
    ``w_value [heads * vdim, rank]`` -> ``[Tq, heads, vdim]``."""
    Tq, heads, dim = q.shape
    T = c.shape[0]
    k = (c @ w_key.T).view(T, heads, dim)
    v = (c @ w_value.T).view(T, heads, -1)
    i = start + torch.arange(Tq)[:, None]
    j = torch.arange(T)[None, :]
    out = torch.zeros(Tq, heads, v.shape[-1], dtype=q.dtype)
    for a in range(heads):
        s = (q[:, a] @ k[:, a].T) * scale
        out[:, a] = torch.softmax(s.masked_fill(j > i, -math.inf), -1) @ v[:, a]
    return out


def mixer(h, W, p, m, eps):
    T = h.shape[0]
    q = (h @ W[p + "q"].T).view(T, m["heads"], m["dim"])
    c = latent(h, W[p + "dkv"], W[p + "dkv.norm"], eps)
    o = latent_attention(q, c, W[p + "uk"], W[p + "uv"], m["scale"]).reshape(T, -1)
    return (o * sigmoid(h @ W[p + "g"].T)) @ W[p + "o"].T


def feed_forward(h, W, p):
    return gelu_erf(h @ W[p + "up"].T) @ W[p + "down"].T


def residual_gate(h, W, name):
    return sigmoid(h @ W[name].T + W[name + ".b"])


def layer(x, W, p, c, eps, mult):
    """Mixer and feed-forward side by side on one stream."""
    h1 = rms(x, eps) * W[p + "norm1"]
    add = mixer(h1, W, p + "mix.", c["mixer"], eps) * residual_gate(h1, W, p + "rg1")
    if c["mlp"] is not None:
        h2 = rms(x, eps) * W[p + "norm2"]
        add = add + feed_forward(h2, W, p + "mlp.") * residual_gate(h2, W, p + "rg2")
    return x + mult * add


def enter_pass(x, x0, w_in, step):
    """First thing in a pass of the loop: stream and embedding mixed, then the vector of the pass."""
    return torch.cat([x, x0], -1) @ w_in.T + step


def run_order(cfg):
    """``(layer, pass entered right before it or None)`` in the order of execution."""
    n, lp = len(cfg["layers"]), cfg.get("loop")
    if lp is None:
        return [(i, None) for i in range(n)]
    order = [(i, None) for i in range(lp["start"])]
    for t in range(lp["times"]):
        order += [(i, t if i == lp["start"] else None) for i in range(lp["start"], lp["stop"])]
    return order + [(i, None) for i in range(lp["stop"], n)]


def soft_cap(z, cap):
    return cap * torch.tanh(z / cap) if cap else z


def forward(cfg, weights, tokens, residuals=None):
    """Logits ``[T, vocab]`` of one sequence; ``residuals``: a list that receives the stream after every layer run."""
    W = {k: v.double() for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x0 = W["embed"][torch.as_tensor(tokens, dtype=torch.int64)]
    x = x0
    for i, t in run_order(cfg):
        if t is not None:
            x = enter_pass(x, x0, W["loop.in"], W["loop.step"][t])
        x = layer(x, W, f"l{i}.", cfg["layers"][i], eps, cfg["residual_mult"])
        if residuals is not None:
            residuals.append(x)
    z = (rms(x, eps) * W["final.norm"]) @ W["head"].T
    return soft_cap(z, cfg.get("logit_softcap"))


def random_checkpoint(cfg, seed=0):
    """Random weights under the checkpoint's names, scaled so that activations stay of order one."""
    g = torch.Generator().manual_seed(seed)
    W = {}

    def put(name, *shape, std=None, base=0.0):
        std = shape[-1] ** -0.5 if std is None else std
        W[name] = base + torch.randn(shape, generator=g, dtype=torch.float64) * std

    width, vocab = cfg["width"], cfg["vocab"]
    put("embed", vocab, width, std=0.7)
    put("head", vocab, width, std=2.0 * width ** -0.5)
    put("final.norm", std=0.1, base=1.2)
    lp = cfg.get("loop")
    if lp is not None:
        put("loop.in", width, 2 * width)
        put("loop.step", lp["times"], width, std=0.4)
    for i, c in enumerate(cfg["layers"]):
        p, m = f"l{i}.", c["mixer"]
        hk, hv, r = m["heads"] * m["dim"], m["heads"] * m["vdim"], m["kv_rank"]
        put(p + "norm1", std=0.1, base=0.8)
        put(p + "mix.q", hk, width, std=2.0 * width ** -0.5)
        put(p + "mix.dkv", r, width)
        put(p + "mix.dkv.norm", r, std=0.2, base=1.0)
        put(p + "mix.uk", hk, r, std=1.5 * r ** -0.5)
        put(p + "mix.uv", hv, r)
        put(p + "mix.g", hv, width)
        put(p + "mix.o", width, hv)
        put(p + "rg1", width, width)
        put(p + "rg1.b", width, std=0.7)
        if c["mlp"] is not None:
            put(p + "norm2", std=0.1, base=1.3)
            put(p + "mlp.up", c["mlp"]["ff"], width)
            put(p + "mlp.down", width, c["mlp"]["ff"], std=1.5 * c["mlp"]["ff"] ** -0.5)
            put(p + "rg2", width, width)
            put(p + "rg2.b", width, std=0.7)
    return {k: v.to(torch.bfloat16) for k, v in W.items()}
