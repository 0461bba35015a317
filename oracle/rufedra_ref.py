"""Plain, slow Rufedra forward pass in torch (float64 by default), one function per mechanism, written from the design's
equations.  Shares no code with the served path: whole sequences, dense masks, one Python step per token in the
recurrences.

Notation: ``x`` residual ``[T, W]``, N_a an RMS norm with weight ``a``.  Per layer

    x <- x + s1 * N_1b(mixer(N_1 x));   x <- x + s2 * N_2b(ff(N_2 x))        (s1, s2 per channel),

and logits = s * head N_final(x).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch

UNIT_EPS = 1e-6


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def unit(x: torch.Tensor) -> torch.Tensor:
    return x / torch.sqrt((x * x).sum(dim=-1, keepdim=True) + UNIT_EPS)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def gelu_tanh(z: torch.Tensor) -> torch.Tensor:
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def causal_conv(x: torch.Tensor, w: torch.Tensor, b: Optional[torch.Tensor] = None) -> torch.Tensor:
    """x ``[T, C]``, w ``[C, taps]`` (last column = the current token), zeros before the start."""
    taps = w.shape[1]
    pad = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x], dim=0)
    y = sum(pad[i:i + x.shape[0]] * w[:, i] for i in range(taps))
    return y if b is None else y + b


# ---- gated delta rule ----------------------------------------------------------------------------------------------------
def delta_rule(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, g: torch.Tensor, beta: torch.Tensor,
               S: Optional[torch.Tensor] = None):
    """q, k ``[T, H, dk]``, v ``[T, H, dv]``, g, beta ``[T, H]`` -> ``(o [T, H, dv], S [H, dk, dv])``."""
    T, H, dk = q.shape
    S = q.new_zeros(H, dk, v.shape[2]) if S is None else S
    out = []
    for t in range(T):
        S = g[t][:, None, None] * S
        u = beta[t][:, None] * (v[t] - torch.einsum("hkv,hk->hv", S, k[t]))
        S = S + k[t][:, :, None] * u[:, None, :]
        out.append(torch.einsum("hkv,hk->hv", S, q[t]))
    return torch.stack(out), S


def delta(h: torch.Tensor, m: dict, t: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    T, H, G, dk, dv = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k, v = (silu(causal_conv(h @ t[n].T, t[n + ".conv"])) for n in ("q", "k", "v"))
    q = unit(q.reshape(T, G, dk)) * dk ** -0.5
    k = unit(k.reshape(T, G, dk))
    of_head = torch.arange(H) // (H // G)
    g = torch.exp(-torch.exp(t["A_log"]) * softplus(h @ t["a"].T + t["dt_bias"]))
    o, _ = delta_rule(q[:, of_head], k[:, of_head], v.reshape(T, H, dv), g, torch.sigmoid(h @ t["b"].T))
    y = (rms(o, eps) * t["norm"]).reshape(T, H * dv) * silu(h @ t["g"].T)
    return y @ t["o"].T


# ---- windowed attention whose values are its raw keys --------------------------------------------------------------------
def rotate_half(x: torch.Tensor, pos: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x ``[T, n, d]``: entries i and i + dims/2 (i < dims/2) are turned by pos * base^(-2i/dims)."""
    half = dims // 2
    f = float(base) ** (-2.0 * torch.arange(half, dtype=torch.float64) / max(dims, 1))
    ang = pos.to(torch.float64)[:, None] * f[None, :]
    c, s = torch.cos(ang).to(x.dtype)[:, None, :], torch.sin(ang).to(x.dtype)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def visible(T: int, window: int) -> torch.Tensor:
    """bool ``[T, T]``: 0 <= i - j < window."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < window)


def softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, mask: torch.Tensor) -> torch.Tensor:
    """q ``[T, H, dk]``, k ``[T, G, dk]``, v ``[T, G, dv]`` -> ``[T, H, dv]``; head h reads kv head h // (H / G)."""
    of_head = torch.arange(q.shape[1]) // (q.shape[1] // k.shape[1])
    s = torch.einsum("ihd,jhd->hij", q, k[:, of_head]) * scale
    p = torch.softmax(s.masked_fill(~mask[None], float("-inf")), dim=-1)
    return torch.einsum("hij,jhd->ihd", p, v[:, of_head])


def key_value_attention(h: torch.Tensor, m: dict, t: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    T, H, G, dk = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    pos = torch.arange(T)
    q = (h @ t["q"].T + t["q.b"]).reshape(T, H, dk)
    k = (h @ t["k"].T + t["k.b"]).reshape(T, G, dk)
    rot = m["rot"]
    qn = rms(rotate_half(q, pos, rot["dims"], rot["base"]), eps)
    kn = rms(rotate_half(k, pos, rot["dims"], rot["base"]), eps)
    o = softmax_attention(qn, kn, k, m["scale"], visible(T, m["mask"]["size"]))
    return (o.reshape(T, H * dk) * torch.sigmoid(h @ t["g"].T)) @ t["o"].T


# ---- selective scan ------------------------------------------------------------------------------------------------------
def selective_scan(x: torch.Tensor, dt: torch.Tensor, A: torch.Tensor, B: torch.Tensor, C: torch.Tensor, D: torch.Tensor,
                   S: Optional[torch.Tensor] = None):
    """x, dt ``[T, I]``, A ``[I, N]``, B, C ``[T, N]``, D ``[I]`` -> ``(y [T, I], S [I, N])``."""
    S = x.new_zeros(A.shape) if S is None else S
    out = []
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out.append(S @ C[t] + D * x[t])
    return torch.stack(out), S


def mamba(h: torch.Tensor, m: dict, t: Dict[str, torch.Tensor]) -> torch.Tensor:
    I, N, r = m["inner"], m["state"], m["dt_rank"]
    xz = h @ t["in"].T
    x = silu(causal_conv(xz[:, :I], t["conv"], t["conv.b"]))
    p = x @ t["x"].T
    dt = softplus(p[:, :r] @ t["dt"].T + t["dt.b"])
    y, _ = selective_scan(x, dt, -torch.exp(t["A_log"]), p[:, r:r + N], p[:, r + N:], t["D"])
    return (y * silu(xz[:, I:])) @ t["o"].T


def parallel(h: torch.Tensor, m: dict, t: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    def part(name):
        return {k[len(name) + 1:]: v for k, v in t.items() if k.startswith(name + ".")}

    left = key_value_attention(h, m["left"], part("left"), eps)
    right = mamba(h, m["right"], part("right"))
    return float(m["left_scale"]) * left + float(m["right_scale"]) * right


# ---- the model -----------------------------------------------------------------------------------------------------------
def feed_forward(h: torch.Tensor, t: Dict[str, torch.Tensor]) -> torch.Tensor:
    return (gelu_tanh(h @ t["gate"].T) * (h @ t["up"].T)) @ t["down"].T


def forward(config: dict, tensors: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64,
            trace: Optional[list] = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one sequence; ``trace`` (a list) receives the residual after every layer."""
    t = {k: (v.to(dtype) if v.is_floating_point() else v) for k, v in tensors.items()}
    eps = float(config["norm"]["eps"])
    x = t["embed"][torch.tensor(tokens)] * float(config["embedding"]["scale"])
    for i, layer in enumerate(config["layers"]):
        lt = {k[len(f"l{i}."):]: v for k, v in t.items() if k.startswith(f"l{i}.")}
        mix = {k[4:]: v for k, v in lt.items() if k.startswith("mix.")}
        mixer = {"delta": delta, "parallel": parallel}[layer["type"]]
        y = mixer(rms(x, eps) * lt["norm1"], layer["mixer"], mix, eps)
        x = x + rms(y, eps) * lt["norm1b"] * lt["ls1"]
        if layer.get("mlp") is not None:
            y = feed_forward(rms(x, eps) * lt["norm2"], {k[4:]: v for k, v in lt.items() if k.startswith("mlp.")})
            x = x + rms(y, eps) * lt["norm2b"] * lt["ls2"]
        if trace is not None:
            trace.append(x.clone())
    return (rms(x, eps) * t["final.norm"]) @ t["head"].T * float(config["logit_scale"])


def greedy(config: dict, tensors: Dict[str, torch.Tensor], prompt: List[int], n_new: int) -> List[int]:
    toks, out = list(prompt), []
    for _ in range(n_new):
        nxt = int(forward(config, tensors, toks)[-1].argmax())
        out.append(nxt)
        toks.append(nxt)
    return out
