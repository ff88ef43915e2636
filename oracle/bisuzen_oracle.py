"""Plain, slow restatement of the Bisuzen decoder in float64 torch on the CPU: one function per mechanism, whole sequences
only (no cache, no state slots, no batching, no chunking), dense masks and token-by-token loops.  It shares no code with
the engine; the GPU tests compare the engine's kernels and steps with it.

`cfg` is the model's config.json as a dict, `weights` maps checkpoint names to tensors.

Notation.  x_t: residual stream at position t (positions count from 0), x_t = embed[token_t] at the start.
rms(v) = v / sqrt(mean(v^2) + eps).  A layer's norm is elementwise, dyt(v) = tanh(a v) w + b with one number a:
    x <- x + mixer(dyt1(x));   x <- x + ff(dyt2(x))     (the second line only if the layer has a feed-forward)
Layers [a, b) run `times` passes in a row on the same weights, every pass with keys / values / state of its own.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_erf(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def dyt(x: torch.Tensor, weights: dict, name: str) -> torch.Tensor:
    a, w, b = (weights[name + s].to(F64) for s in (".alpha", "", ".b"))
    return torch.tanh(a * x) * w + b


# ------------------------------------------------------------------------------------------------ attention
def rotate_pairs(x: torch.Tensor, rot: dict) -> torch.Tensor:
    """x [T, heads, d]: entry 2i of the first `dims` turns together with entry 2i + 1 by the angle t * base^(-2i / dims)."""
    dims, base = int(rot["dims"]), float(rot["base"])
    f = torch.tensor([base ** (-2.0 * i / dims) for i in range(dims // 2)], dtype=F64)
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * f[None, :]
    c, s = ang.cos()[:, None, :], ang.sin()[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def window_mask(T: int, size: int, keep_first: int) -> torch.Tensor:
    """[T, T] bool: query i sees key j <= i if it is one of the last `size` positions or one of the first `keep_first`."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def chunk_mask(T: int, size: int) -> torch.Tensor:
    """[T, T] bool: query i sees key j <= i of its own chunk of `size` positions."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (torch.div(i, size, rounding_mode="floor") == torch.div(j, size, rounding_mode="floor"))


def attend(q, k, v, mask, scale: float, sink=None) -> torch.Tensor:
    """q [T, H, d], k [T, G, d], v [T, G, dv] -> [T, H, dv]; sink [H]: one more term exp(sink_h) in the denominator."""
    T, H, G = q.shape[0], q.shape[1], k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for h in range(H):
        g = h // (H // G)
        s = (q[:, h] @ k[:, g].T * scale).masked_fill(~mask, -math.inf)
        mx = s.max(-1, keepdim=True).values
        if sink is not None:
            mx = torch.maximum(mx, sink[h])
        e = torch.exp(s - mx)
        den = e.sum(-1, keepdim=True)
        if sink is not None:
            den = den + torch.exp(sink[h] - mx)
        out[:, h] = e @ v[:, g] / den
    return out


def window_attention(h: torch.Tensor, w: dict, m: dict) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rotate_pairs((h @ w["q"].T + w["q.b"]).view(T, H, d), m["rot"])
    k = rotate_pairs((h @ w["k"].T + w["k.b"]).view(T, G, d), m["rot"])
    v = (h @ w["v"].T + w["v.b"]).view(T, G, dv)
    mask = window_mask(T, int(m["mask"]["size"]), int(m["mask"].get("keep_first", 0)))
    o = attend(q, k, v, mask, float(m["scale"]), w["sink"])
    return o.reshape(T, H * dv) @ w["o"].T + w["o.b"]


def chunked_attention(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    q = rms((h @ w["q"].T).view(T, H, d), eps)
    k = rms((h @ w["k"].T).view(T, G, d), eps)
    v = (h @ w["v"].T).view(T, G, dv)
    o = attend(q, k, v, chunk_mask(T, int(m["mask"]["size"])), float(m["scale"]))
    return o.reshape(T, H * dv) @ w["o"].T


# ------------------------------------------------------------------------------------------------ lightning attention
def lightning(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    """Per head a matrix S [dim, vdim]: S <- decay S + k v^T, o = S^T q; all heads of o normed together, gated."""
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = silu(h @ w["q"].T).view(T, H, d)
    k = silu(h @ w["k"].T).view(T, H, d)
    v = silu(h @ w["v"].T).view(T, H, dv)
    decay = torch.tensor([float(x) for x in m["decay"]], dtype=F64)
    S = torch.zeros(H, d, dv, dtype=F64)
    out = torch.zeros(T, H, dv, dtype=F64)
    for t in range(T):
        S = decay[:, None, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    y = rms(out.reshape(T, H * dv), eps) * w["norm"] * torch.sigmoid(h @ w["g"].T)
    return y @ w["o"].T


def parallel(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    a = window_attention(h, sub(w, "left."), m["left"])
    b = lightning(h, sub(w, "right."), m["right"], eps)
    return 0.5 * (rms(a, eps) * w["left.out"] + rms(b, eps) * w["right.out"])


# ------------------------------------------------------------------------------------------------ feed-forward
def dense_ff(h: torch.Tensor, w: dict) -> torch.Tensor:
    return (gelu_tanh(h @ w["gate"].T) * (h @ w["up"].T)) @ w["down"].T


def route(z: torch.Tensor, correction: torch.Tensor, r: dict) -> list[list[tuple[int, float]]]:
    """[(output, weight)] of every row of router logits z [T, experts + identity]."""
    n, top = z.shape[1], int(r["top"])
    groups = r.get("groups") or {"count": 1, "keep": 1}
    count, keep = int(groups["count"]), int(groups["keep"])
    per = n // count
    out = []
    for s in torch.softmax(z, -1):
        c = s + correction
        best = sorted(range(count), key=lambda g: -float(c[g * per : (g + 1) * per].max()))[:keep]
        allowed = [e for e in range(n) if e // per in best]
        chosen = sorted(allowed, key=lambda e: -float(c[e]))[:top]
        tot = sum(float(s[e]) for e in chosen) + 1e-20
        out.append([(e, float(s[e]) / tot) for e in chosen])
    return out


def moe_ff(h: torch.Tensor, w: dict, r: dict) -> torch.Tensor:
    out = torch.zeros_like(h)
    for t, pairs in enumerate(route(h @ w["router"].T, w["correction"], r)):
        for e, p in pairs:
            y = h[t] if e >= int(r["experts"]) else w[f"e{e}.down"] @ gelu_erf(w[f"e{e}.up"] @ h[t])
            out[t] += p * y
    return out


# ------------------------------------------------------------------------------------------------ the stack
def sub(weights: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v.to(F64) for k, v in weights.items() if k.startswith(prefix)}


def layer_runs(cfg: dict) -> list[int]:
    n = len(cfg["layers"])
    loop = cfg.get("loop") or {"start": 0, "stop": 0, "times": 1}
    a, b, times = int(loop["start"]), int(loop["stop"]), int(loop["times"])
    if b <= a:
        return list(range(n))
    return list(range(a)) + list(range(a, b)) * times + list(range(b, n))


def forward(cfg: dict, weights: dict, tokens: list[int], layers_out: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of the whole sequence; `layers_out` collects the stream after every layer run."""
    eps = float(cfg["norm"]["eps"])
    x = weights["embed"].to(F64)[torch.tensor(tokens, dtype=torch.long)]
    for i in layer_runs(cfg):
        L, p = cfg["layers"][i], f"l{i}."
        mix = parallel if L["type"] == "parallel" else chunked_attention
        x = x + mix(dyt(x, weights, p + "norm1"), sub(weights, p + "mix."), L["mixer"], eps)
        mlp = L.get("mlp")
        if mlp is not None:
            h, w = dyt(x, weights, p + "norm2"), sub(weights, p + "mlp.")
            x = x + (dense_ff(h, w) if mlp["kind"] == "dense" else moe_ff(h, w, mlp["router"]))
        if layers_out is not None:
            layers_out.append(x.clone())
    return dyt(x, weights, "final.norm") @ weights["head"].to(F64).T * float(cfg.get("logit_scale", 1.0))


def greedy(cfg: dict, weights: dict, prompt: list[int], n_new: int) -> list[int]:
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]
