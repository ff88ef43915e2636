"""Plain, slow restatement of the Ludelix decoder in float64 torch on the CPU: one function per mechanism, whole sequences
only (no cache, no state slots, no batching, no chunking), dense masks and token-by-token loops.  It shares no code with
the engine; the GPU tests compare the engine's kernels and steps with it.

`cfg` is the model's config.json as a dict, `weights` maps checkpoint names to tensors.

Notation.  x_t: residual stream at position t (positions count from 0), x_t = embed[token_t] at the start.
rms(v) = v / sqrt(mean(v^2) + eps).  Layers are pre-normed with plain weights:
    x <- x + mixer(rms(x) * norm1);   x <- x + ff(rms(x) * norm2)     (the second line only if the layer has a feed-forward)
Logits read the embedding table.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(v: torch.Tensor, eps: float) -> torch.Tensor:
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


# ------------------------------------------------------------------------------------------------ rotary positions
def plain_freqs(rot: dict) -> list[float]:
    dims, base = int(rot["dims"]), float(rot["base"])
    return [base ** (-2.0 * i / dims) for i in range(dims // 2)]


def banded_freqs(rot: dict) -> list[float]:
    """Frequencies whose wavelength is long against `original` positions are divided by `factor`, short ones stay, the
    ones between are blended by where original / wavelength lies between `low` and `high` (Llama 3.1's rule)."""
    s = rot["scaling"]
    factor, low, high, original = (float(s[k]) for k in ("factor", "low", "high", "original"))
    out = []
    for f in plain_freqs(rot):
        wave = 2.0 * math.pi / f
        if wave < original / high:
            out.append(f)
        elif wave > original / low:
            out.append(f / factor)
        else:
            t = (original / wave - low) / (high - low)
            out.append((1.0 - t) * f / factor + t * f)
    return out


def yarn_freqs(rot: dict) -> tuple[list[float], float]:
    """(frequencies, factor on cosine and sine) under YaRN."""
    s, dims, base = rot["scaling"], int(rot["dims"]), float(rot["base"])
    factor, original = float(s["factor"]), float(s["original"])

    def turns_at(t):
        return dims * math.log(original / (2.0 * math.pi * t)) / (2.0 * math.log(base))

    lo = max(math.floor(turns_at(float(s["fast"]))), 0)
    hi = min(math.ceil(turns_at(float(s["slow"]))), dims - 1)
    out = []
    for i, f in enumerate(plain_freqs(rot)):
        r = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(f / factor * r + f * (1.0 - r))
    return out, 0.1 * math.log(factor) + 1.0


def rotate(x: torch.Tensor, freqs: list[float], interleaved: bool, mag: float = 1.0) -> torch.Tensor:
    """x [T, heads, d]; pairs (2i, 2i + 1) or (i, i + n) of the first 2 n = 2 len(freqs) entries turn by t * freqs[i]."""
    n = len(freqs)
    ang = torch.arange(x.shape[0], dtype=F64)[:, None] * torch.tensor(freqs, dtype=F64)[None, :]
    c, s = mag * ang.cos()[:, None, :], mag * ang.sin()[:, None, :]
    a = slice(0, 2 * n, 2) if interleaved else slice(0, n)
    b = slice(1, 2 * n, 2) if interleaved else slice(n, 2 * n)
    out = x.clone()
    out[..., a] = x[..., a] * c - x[..., b] * s
    out[..., b] = x[..., b] * c + x[..., a] * s
    return out


# ------------------------------------------------------------------------------------------------ attention
def window_mask(T: int, size: int) -> torch.Tensor:
    """[T, T] bool: query i sees the `size` keys that end with its own."""
    i, j = torch.arange(T)[:, None], torch.arange(T)[None, :]
    return (j <= i) & (i - j < size)


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


def shared_attention(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    """Sliding-window attention with one projection for keys and values: the value is its biased output, the key that output normed and turned."""
    T = h.shape[0]
    H, G, d = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    q, k = h @ w["q"].T + w["q.b"], h @ w["k"].T + w["k.b"]
    v = k.view(T, G, d)
    f = banded_freqs(m["rot"])
    q = rotate((rms(q, eps) * w["q.norm"]).view(T, H, d), f, True)
    k = rotate((rms(k, eps) * w["k.norm"]).view(T, G, d), f, True)
    o = attend(q, k, v, window_mask(T, int(m["mask"]["size"])), float(m["scale"]), w["sink"])
    return o.reshape(T, H * d) @ w["o"].T


def gated_chunk_attention(h: torch.Tensor, w: dict, m: dict) -> torch.Tensor:
    T = h.shape[0]
    H, G, d, dv = int(m["heads"]), int(m["kv_heads"]), int(m["dim"]), int(m["vdim"])
    f, mag = yarn_freqs(m["rot"])
    q = rotate((h @ w["q"].T).view(T, H, d), f, False, mag)
    k = rotate((h @ w["k"].T).view(T, G, d), f, False, mag)
    v = (h @ w["v"].T).view(T, G, dv)
    o = attend(q, k, v, chunk_mask(T, int(m["mask"]["size"])), float(m["scale"]))
    o = o * torch.sigmoid(h @ w["g"].T)[:, :, None]
    return o.reshape(T, H * dv) @ w["o"].T


# ------------------------------------------------------------------------------------------------ recurrent mixers
def outer_memory(q, k, v, decay) -> torch.Tensor:
    """q, k [T, H, d], v [T, H, dv], decay [T, H, d] (per key channel): S <- diag(decay) S + k v^T, o = S^T q."""
    T, H, d = q.shape
    S = torch.zeros(H, d, v.shape[-1], dtype=F64)
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for t in range(T):
        S = decay[t][:, :, None] * S + k[t][:, :, None] * v[t][:, None, :]
        out[t] = torch.einsum("hdv,hd->hv", S, q[t])
    return out


def retention(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    f = plain_freqs(m["rot"])
    q = rotate((h @ w["q"].T).view(T, H, d), f, False)
    k = rotate((h @ w["k"].T).view(T, H, d), f, False) * d ** -0.5
    v = (h @ w["v"].T).view(T, H, dv)
    decay = torch.tensor([float(x) for x in m["decay"]], dtype=F64)[None, :, None].expand(T, H, d)
    o = rms(outer_memory(q, k, v, decay), eps).reshape(T, H * dv)
    return (o * silu(h @ w["g"].T)) @ w["o"].T


def gated_linear(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    T = h.shape[0]
    H, d, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
    q = (h @ w["q"].T).view(T, H, d) * d ** -0.5
    k = (h @ w["k"].T).view(T, H, d)
    v = (h @ w["v"].T).view(T, H, dv)
    z = h @ w["a1"].T @ w["a2"].T + w["a2.b"]
    decay = (torch.sigmoid(z) ** (1.0 / float(m["tau"]))).view(T, H, d)
    o = (rms(outer_memory(q, k, v, decay), eps) * w["norm"]).reshape(T, H * dv)
    return (o * silu(h @ w["g"].T)) @ w["o"].T


def parallel(h: torch.Tensor, w: dict, m: dict, eps: float) -> torch.Tensor:
    return (float(m["left_scale"]) * gated_chunk_attention(h, sub(w, "left."), m["left"])
            + float(m["right_scale"]) * retention(h, sub(w, "right."), m["right"], eps))


# ------------------------------------------------------------------------------------------------ feed-forward
def dense_ff(h: torch.Tensor, w: dict) -> torch.Tensor:
    return torch.relu(h @ w["up"].T) ** 2 @ w["down"].T


def expert(h: torch.Tensor, w: dict, name: str) -> torch.Tensor:
    return (silu(h @ w[name + ".gate"].T) * (h @ w[name + ".up"].T)) @ w[name + ".down"].T


def table_ff(h: torch.Tensor, w: dict, mlp: dict, tokens: list[int]) -> torch.Tensor:
    """The token id picks its experts from a table, each with weight 1 / top; a shared expert under a sigmoid is added."""
    out = torch.zeros_like(h)
    for t, tok in enumerate(tokens):
        chosen = w["table"][tok].long().tolist()
        for e in chosen:
            out[t] += expert(h[t], w, f"e{e}") / len(chosen)
    if mlp.get("shared"):
        out = out + torch.sigmoid(h @ w["shared.sg"].T) * expert(h, w, "shared")
    return out


# ------------------------------------------------------------------------------------------------ the stack
def sub(weights: dict, prefix: str) -> dict:
    return {k[len(prefix):]: v.to(F64) for k, v in weights.items() if k.startswith(prefix)}


MIXERS = {"parallel": parallel, "gla": gated_linear, "attention": shared_attention}


def forward(cfg: dict, weights: dict, tokens: list[int], layers_out: list | None = None) -> torch.Tensor:
    """Logits [T, vocab] of the whole sequence; `layers_out` collects the stream after every layer."""
    eps, emb = float(cfg["norm"]["eps"]), weights["embed"].to(F64)

    def norm(x, name):
        return rms(x, eps) * weights[name].to(F64)

    x = emb[torch.tensor(tokens, dtype=torch.long)]
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        x = x + MIXERS[L["type"]](norm(x, p + "norm1"), sub(weights, p + "mix."), L["mixer"], eps)
        mlp = L.get("mlp")
        if mlp is not None:
            h, w = norm(x, p + "norm2"), sub(weights, p + "mlp.")
            x = x + (dense_ff(h, w) if mlp["kind"] == "dense" else table_ff(h, w, mlp, tokens))
        if layers_out is not None:
            layers_out.append(x.clone())
    return norm(x, "final.norm") @ emb.T


def greedy(cfg: dict, weights: dict, prompt: list[int], n_new: int) -> list[int]:
    toks = list(prompt)
    for _ in range(n_new):
        toks.append(int(forward(cfg, weights, toks)[-1].argmax()))
    return toks[len(prompt):]
