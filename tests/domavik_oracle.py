"""Plain, slow statement of the Domavik decoder in float64: one function per mechanism, token by token where the design is
recurrent, no batching, no cache.  It is written from the equations and imports nothing of the package, so the tests
compare two independent programs.  ``weights`` maps checkpoint names to tensors, ``cfg`` is the parsed config.json."""
from __future__ import annotations

import math

import torch


def layer_norm(x, w, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def gelu_tanh(z):
    return 0.5 * z * (1 + torch.tanh(math.sqrt(2 / math.pi) * (z + 0.044715 * z ** 3)))


def window_attention(q, k, v, scale, size, keep_first, start=0):
    """``q [Tq, H, dk]`` at positions ``start ..``, ``k [T, G, dk]``, ``v [T, G, dv]`` -> ``[Tq, H, dv]``."""
    Tq, H, _ = q.shape
    T, G, _ = k.shape
    out = torch.zeros(Tq, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        slope = 2.0 ** (-8.0 * (h + 1) / H)
        for t in range(Tq):
            i = start + t
            seen = [j for j in range(min(i + 1, T)) if i - j < size or j < keep_first]
            s = torch.stack([(q[t, h] * k[j, g]).sum() * scale - slope * (i - j) for j in seen])
            p = torch.softmax(s, 0)
            out[t, h] = sum(p[n] * v[j, g] for n, j in enumerate(seen))
    return out


def window_attention_fast(q, k, v, scale, size, keep_first):
    """The same by dense matrices (whole prompts of some hundred tokens)."""
    T, H, _ = q.shape
    G = k.shape[1]
    i = torch.arange(T, dtype=q.dtype)[:, None]
    j = torch.arange(T, dtype=q.dtype)[None, :]
    seen = (j <= i) & ((i - j < size) | (j < keep_first))
    out = torch.zeros(T, H, v.shape[-1], dtype=q.dtype)
    for h in range(H):
        g = h // (H // G)
        s = q[:, h] @ k[:, g].T * scale - 2.0 ** (-8.0 * (h + 1) / H) * (i - j)
        out[:, h] = torch.softmax(s.masked_fill(~seen, -math.inf), -1) @ v[:, g]
    return out


def gated_linear(q, k, v, z, tau, state=None):
    """``q, k, z [T, h, dk]``, ``v [T, h, dv]``; returns outputs ``[T, h, dv]`` and the final state ``[h, dk, dv]``."""
    T, h, dk = q.shape
    S = torch.zeros(h, dk, v.shape[-1], dtype=q.dtype) if state is None else state.clone()
    out = []
    for t in range(T):
        alpha = torch.sigmoid(z[t]) ** (1.0 / tau)
        S = alpha[:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out.append((S * q[t][:, :, None]).sum(1))
    return torch.stack(out), S


def matrix_memory(q, k, v, zi, zf, cap, state=None):
    """``q, k [T, h, dk]``, ``v [T, h, dv]``, ``zi, zf [T, h]`` gate pre-activations with their biases; returns outputs
    and the final ``(S, n, m)``."""
    T, h, dk = q.shape
    if state is None:
        S = torch.zeros(h, dk, v.shape[-1], dtype=q.dtype)
        n = torch.zeros(h, dk, dtype=q.dtype)
        m = torch.zeros(h, dtype=q.dtype)
    else:
        S, n, m = (x.clone() for x in state)
    out = []
    for t in range(T):
        i = cap * torch.tanh(zi[t] / cap)
        f = torch.nn.functional.logsigmoid(cap * torch.tanh(zf[t] / cap))
        m_new = torch.maximum(f + m, i)
        keep, put = torch.exp(f + m - m_new), torch.exp(i - m_new)
        S = keep[:, None, None] * S + put[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + put[:, None] * k[t]
        m = m_new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append((S * q[t][:, :, None]).sum(1) / den[:, None])
    return torch.stack(out), (S, n, m)


def attention_mixer(x, W, p, c):
    T, H, G = x.shape[0], c["heads"], c["kv_heads"]
    q = (x @ W[p + "q"].T).view(T, H, c["dim"])
    k = (x @ W[p + "k"].T).view(T, G, c["dim"])
    v = (x @ W[p + "v"].T).view(T, G, c["vdim"])
    o = window_attention_fast(q, k, v, c["scale"], c["mask"]["size"], c["mask"]["keep_first"])
    return o.reshape(T, -1) @ W[p + "o"].T


def gated_linear_mixer(x, W, p, c, eps):
    T, h, dk, dv = x.shape[0], c["heads"], c["dim"], c["vdim"]
    q = (x @ W[p + "q"].T).view(T, h, dk) * dk ** -0.5
    k = (x @ W[p + "k"].T).view(T, h, dk)
    v = (x @ W[p + "v"].T).view(T, h, dv)
    z = (x @ W[p + "a1"].T @ W[p + "a2"].T + W[p + "a2.b"]).view(T, h, dk)
    o, _ = gated_linear(q, k, v, z, c["tau"])
    o = (rms(o, eps) * W[p + "norm"]).reshape(T, -1)
    g = x @ W[p + "g"].T
    return (o * g * torch.sigmoid(g)) @ W[p + "o"].T


def matrix_memory_mixer(x, W, p, c, eps):
    T, h, dk, dv = x.shape[0], c["heads"], c["dim"], c["vdim"]
    q = (x @ W[p + "q"].T).view(T, h, dk) * dk ** -0.5
    k = (x @ W[p + "k"].T).view(T, h, dk)
    v = (x @ W[p + "v"].T).view(T, h, dv)
    zi = x @ W[p + "i"].T + W[p + "i.b"]
    zf = x @ W[p + "f"].T + W[p + "f.b"]
    o, _ = matrix_memory(q, k, v, zi, zf, c["gate_cap"])
    o = rms(o, eps).reshape(T, -1) * W[p + "norm"]
    return (o * torch.sigmoid(x @ W[p + "g"].T)) @ W[p + "o"].T


def mixer(x, W, p, layer, eps):
    c = layer["mixer"]
    if layer["type"] == "mlstm":
        return matrix_memory_mixer(x, W, p, c, eps)
    assert layer["type"] == "parallel"
    return c["left_scale"] * attention_mixer(x, W, p + "left.", c["left"]) + \
        c["right_scale"] * gated_linear_mixer(x, W, p + "right.", c["right"], eps)


def feed_forward(x, W, p):
    return (gelu_tanh(x @ W[p + "gate"].T) * (x @ W[p + "up"].T)) @ W[p + "down"].T


def forward(cfg, weights, tokens, residuals=None):
    """Logits ``[T, vocab]`` of one sequence; ``residuals``: a list that receives the stream after every layer."""
    W = {k: v.double() for k, v in weights.items()}
    eps = cfg["norm"]["eps"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.int64)] * cfg["embedding"]["scale"]
    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + mixer(layer_norm(x, W[p + "norm1"], eps), W, p + "mix.", layer, eps)
        if layer["mlp"] is not None:
            x = x + feed_forward(layer_norm(x, W[p + "norm2"], eps), W, p + "mlp.")
        if residuals is not None:
            residuals.append(x)
    z = layer_norm(x, W["final.norm"], eps) @ W["head"].T
    cap = cfg["logit_softcap"]
    return cap * torch.tanh(z / cap)


def random_checkpoint(cfg, seed=0, gate_rank=8):
    """Random weights under the checkpoint's names, scaled so that activations stay of order one."""
    g = torch.Generator().manual_seed(seed)
    W = {}

    def put(name, *shape, std=None, base=0.0):
        W[name] = base + torch.randn(*shape, generator=g, dtype=torch.float64) * (shape[-1] ** -0.5 if std is None else std)

    width, vocab = cfg["width"], cfg["vocab"]
    put("embed", vocab, width, std=0.5)
    put("head", vocab, width, std=2.0 * width ** -0.5)
    put("final.norm", width, std=0.1, base=1.0)

    def branch(p, c, kind):
        hk, hv = c["heads"] * c["dim"], c["heads"] * c["vdim"]
        gk, gv = c.get("kv_heads", c["heads"]) * c["dim"], c.get("kv_heads", c["heads"]) * c["vdim"]
        put(p + "q", hk, width, std=1.5 * width ** -0.5)
        put(p + "k", gk, width, std=1.5 * width ** -0.5)
        put(p + "v", gv, width)
        put(p + "o", width, hv)
        if kind == "attention":
            return
        put(p + "g", hv, width)
        if kind == "gla":
            put(p + "norm", c["vdim"], std=0.1, base=1.0)
            put(p + "a1", gate_rank, width)
            put(p + "a2", hk, gate_rank, std=1.0)
            put(p + "a2.b", hk, std=1.5)
        else:
            put(p + "norm", hv, std=0.1, base=1.0)
            for n, b in (("i", -1.0), ("f", 3.0)):
                put(p + n, c["heads"], width)
                put(p + n + ".b", c["heads"], std=1.0, base=b)

    for i, layer in enumerate(cfg["layers"]):
        p = f"l{i}."
        put(p + "norm1", width, std=0.1, base=1.0)
        if layer["type"] == "mlstm":
            branch(p + "mix.", layer["mixer"], "mlstm")
        else:
            branch(p + "mix.left.", layer["mixer"]["left"], "attention")
            branch(p + "mix.right.", layer["mixer"]["right"], "gla")
        if layer["mlp"] is not None:
            ff = layer["mlp"]["ff"]
            put(p + "norm2", width, std=0.1, base=1.0)
            put(p + "mlp.gate", ff, width)
            put(p + "mlp.up", ff, width)
            put(p + "mlp.down", width, ff)
    return {k: v.to(torch.bfloat16) for k, v in W.items()}
