"""Plain, slow Zuderax forward pass in torch (float64 by default), one function per mechanism, written from the design's
equations.  Shares no code with the served path: whole sequences, dense masks, one Python step per token in the
recurrences, a loop over experts.

Notation: ``x`` residual ``[T, W]``.  Per layer

    x <- x + mixer(D1(x));   x <- x + ff(D2(x))        with D(x) = tanh(alpha x) * w + b, alpha a scalar,

and logits = s * head D_final(x).
"""
from __future__ import annotations

import math
from typing import Dict, List, Optional

import torch


def rms(x: torch.Tensor, eps: float) -> torch.Tensor:
    return x / torch.sqrt((x * x).mean(dim=-1, keepdim=True) + eps)


def silu(z: torch.Tensor) -> torch.Tensor:
    return z * torch.sigmoid(z)


def softplus(z: torch.Tensor) -> torch.Tensor:
    return torch.clamp(z, min=0) + torch.log1p(torch.exp(-z.abs()))


def dyn_tanh(x: torch.Tensor, alpha: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    return torch.tanh(alpha * x) * w + b


# ---- latent attention ------------------------------------------------------------------------------------------------
def rotate_half(x: torch.Tensor, pos: torch.Tensor, dims: int, base: float) -> torch.Tensor:
    """x ``[T, ..., d]``: entries i and i + dims/2 (i < dims/2) are turned by pos * base^(-2i/dims)."""
    half = dims // 2
    f = float(base) ** (-2.0 * torch.arange(half, dtype=torch.float64) / dims)
    ang = pos.to(torch.float64)[:, None] * f[None, :]
    shape = [x.shape[0]] + [1] * (x.dim() - 2) + [half]
    c, s = torch.cos(ang).to(x.dtype).reshape(shape), torch.sin(ang).to(x.dtype).reshape(shape)
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def visible(T: int, window: int) -> torch.Tensor:
    """bool ``[T, T]``: 0 <= i - j < window (window 0: every j <= i)."""
    d = torch.arange(T)[:, None] - torch.arange(T)[None, :]
    return (d >= 0) & (d < window) if window > 0 else d >= 0


def softmax_attention(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, scale: float, mask: torch.Tensor) -> torch.Tensor:
    """q, k ``[T, H, dk]``, v ``[T, H, dv]`` -> ``[T, H, dv]``."""
    s = torch.einsum("ihd,jhd->hij", q, k) * scale
    p = torch.softmax(s.masked_fill(~mask[None], float("-inf")), dim=-1)
    return torch.einsum("hij,jhd->ihd", p, v)


def latent_attention(h: torch.Tensor, m: dict, t: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    T, H, dn, dr, dv, r = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    pos = torch.arange(T)
    q = (h @ t["q"].T).reshape(T, H, dn + dr)
    d = h @ t["dkv"].T
    c = rms(d[:, :r], eps) * t["dkv.norm"]
    rot = m["rot"]
    k_rot = rotate_half(d[:, r:], pos, rot["dims"], rot["base"])
    q_rot = rotate_half(q[..., dn:], pos, rot["dims"], rot["base"])
    k = torch.cat([(c @ t["uk"].T).reshape(T, H, dn), k_rot[:, None, :].expand(T, H, dr)], dim=-1)
    v = (c @ t["uv"].T).reshape(T, H, dv)
    o = softmax_attention(torch.cat([q[..., :dn], q_rot], dim=-1), k, v, m["scale"], visible(T, m["mask"]["size"]))
    return o.reshape(T, H * dv) @ t["o"].T


# ---- mLSTM -------------------------------------------------------------------------------------------------------------
def capped_gates(zi: torch.Tensor, zf: torch.Tensor, cap: float):
    """``(i, f)``: log input gate cap tanh(zi / cap), log forget gate log sigmoid(cap tanh(zf / cap))."""
    return cap * torch.tanh(zi / cap), -softplus(-cap * torch.tanh(zf / cap))


def matrix_memory(q: torch.Tensor, k: torch.Tensor, v: torch.Tensor, i: torch.Tensor, f: torch.Tensor,
                  state: Optional[tuple] = None):
    """q, k ``[T, H, dk]``, v ``[T, H, dv]``, i, f ``[T, H]`` -> ``(o [T, H, dv], (S, n, m))``; the running maximum starts
    at 0."""
    T, H, dk = q.shape
    if state is None:
        state = (q.new_zeros(H, dk, v.shape[2]), q.new_zeros(H, dk), q.new_zeros(H))
    S, n, m = state
    out = []
    for t in range(T):
        new = torch.maximum(f[t] + m, i[t])
        keep, write = torch.exp(f[t] + m - new), torch.exp(i[t] - new)
        S = keep[:, None, None] * S + write[:, None, None] * k[t][:, :, None] * v[t][:, None, :]
        n = keep[:, None] * n + write[:, None] * k[t]
        m = new
        den = torch.maximum((n * q[t]).sum(-1).abs(), torch.exp(-m)) + 1e-6
        out.append(torch.einsum("hkv,hk->hv", S, q[t]) / den[:, None])
    return torch.stack(out), (S, n, m)


def mlstm(h: torch.Tensor, m: dict, t: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    T, H, dk, dv = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = (h @ t["q"].T).reshape(T, H, dk) * dk ** -0.5
    k, v = (h @ t["k"].T).reshape(T, H, dk), (h @ t["v"].T).reshape(T, H, dv)
    i, f = capped_gates(h @ t["i"].T + t["i.b"], h @ t["f"].T + t["f.b"], float(m["gate_cap"]))
    o, _ = matrix_memory(q, k, v, i, f)
    y = rms(o, eps).reshape(T, H * dv) * t["norm"] * torch.sigmoid(h @ t["g"].T)
    return y @ t["o"].T


# ---- Mamba-2 -----------------------------------------------------------------------------------------------------------
def causal_conv(x: torch.Tensor, w: torch.Tensor, b: torch.Tensor) -> torch.Tensor:
    """x ``[T, C]``, w ``[C, taps]`` (last column = the current token), zeros before the start."""
    taps = w.shape[1]
    pad = torch.cat([x.new_zeros(taps - 1, x.shape[1]), x], dim=0)
    return sum(pad[i:i + x.shape[0]] * w[:, i] for i in range(taps)) + b


def state_space(x: torch.Tensor, B: torch.Tensor, C: torch.Tensor, dt: torch.Tensor, a_log: torch.Tensor, D: torch.Tensor,
                S: Optional[torch.Tensor] = None):
    """x ``[T, H, dv]``, B, C ``[T, G, N]``, dt ``[T, H]`` (after softplus) -> ``(y [T, H, dv], S [H, N, dv])``."""
    T, H, dv = x.shape
    G, N = B.shape[1:]
    of = torch.arange(H) // (H // G)
    if S is None:
        S = x.new_zeros(H, N, dv)
    out = []
    for t in range(T):
        keep = torch.exp(-torch.exp(a_log) * dt[t])
        S = keep[:, None, None] * S + (dt[t][:, None] * B[t][of])[:, :, None] * x[t][:, None, :]
        out.append(torch.einsum("hnv,hn->hv", S, C[t][of]) + D[:, None] * x[t])
    return torch.stack(out), S


def mamba2(h: torch.Tensor, m: dict, t: Dict[str, torch.Tensor], eps: float) -> torch.Tensor:
    T, H, dv, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * dv
    p = h @ t["in"].T
    z, xbc, dt = p[:, :inner], p[:, inner:2 * inner + 2 * G * N], p[:, 2 * inner + 2 * G * N:]
    xbc = silu(causal_conv(xbc, t["conv"], t["conv.b"]))
    x = xbc[:, :inner].reshape(T, H, dv)
    B, C = xbc[:, inner:inner + G * N].reshape(T, G, N), xbc[:, inner + G * N:].reshape(T, G, N)
    y, _ = state_space(x, B, C, softplus(dt + t["dt_bias"]), t["A_log"], t["D"])
    y = y.reshape(T, inner) * silu(z)
    y = rms(y.reshape(T, m["norm_groups"], -1), eps).reshape(T, inner) * t["norm"]
    return y @ t["o"].T


# ---- feed-forward ------------------------------------------------------------------------------------------------------
def glu(h: torch.Tensor, t: Dict[str, torch.Tensor], pre: str = "") -> torch.Tensor:
    return (silu(h @ t[pre + "gate"].T) * (h @ t[pre + "up"].T)) @ t[pre + "down"].T


def route(z: torch.Tensor, correction: Optional[torch.Tensor], top: int, groups: int, keep: int, scale: float):
    """``(ids [T, top], weights [T, top])``: sigmoid scores; choice by score + correction inside the ``keep`` groups whose
    two best choice scores have the largest sum; weights = scale * score."""
    s = torch.sigmoid(z)
    c = s if correction is None else s + correction
    per = z.shape[1] // groups
    best = c.reshape(-1, groups, per).sort(dim=-1, descending=True).values[..., :2].sum(-1)
    kept = best.sort(dim=-1, descending=True, stable=True).indices[:, :keep]
    ok = torch.zeros_like(best, dtype=torch.bool).scatter_(1, kept, True).repeat_interleave(per, dim=1)
    ids = c.masked_fill(~ok, float("-inf")).sort(dim=-1, descending=True, stable=True).indices[:, :top]
    return ids, s.gather(1, ids) * scale


def moe(h: torch.Tensor, spec: dict, t: Dict[str, torch.Tensor]) -> torch.Tensor:
    r = spec["router"]
    g = r.get("groups") or {"count": 1, "keep": 1}
    ids, w = route(h @ t["router"].T, t.get("correction"), r["top"], g["count"], g["keep"], float(r.get("scale", 1.0)))
    out = torch.zeros_like(h)
    for n in range(h.shape[0]):
        for e, we in zip(ids[n].tolist(), w[n]):
            out[n] += we * glu(h[n:n + 1], t, f"e{e}.")[0]
    if spec.get("shared"):
        out = out + torch.sigmoid(h @ t["shared.sg"].T) * glu(h, t, "shared.")
    return out


# ---- the model ---------------------------------------------------------------------------------------------------------
MIXERS = {"latent_attention": latent_attention, "mlstm": mlstm, "mamba2": mamba2}


def forward(config: dict, tensors: Dict[str, torch.Tensor], tokens: List[int], dtype=torch.float64,
            trace: Optional[list] = None) -> torch.Tensor:
    """Logits ``[T, vocab]`` of one whole sequence; ``trace`` receives the residual after every layer."""
    w = {k: v.to(dtype) if v.is_floating_point() else v for k, v in tensors.items()}
    eps = float(config["norm"]["eps"])
    x = w["embed"][torch.tensor(tokens)]

    def norm(x, name):
        return dyn_tanh(x, w[name + ".alpha"], w[name], w[name + ".b"])

    for i, layer in enumerate(config["layers"]):
        src = layer.get("weights_of")
        pre = f"l{i if src is None else src}."
        mix = {k[len(pre) + 4:]: v for k, v in w.items() if k.startswith(pre + "mix.")}
        x = x + MIXERS[layer["type"]](norm(x, pre + "norm1"), layer["mixer"], mix, eps)
        mlp = layer.get("mlp")
        if mlp is not None:
            t = {k[len(pre) + 4:]: v for k, v in w.items() if k.startswith(pre + "mlp.")}
            h = norm(x, pre + "norm2")
            x = x + (moe(h, mlp, t) if mlp["kind"] == "moe" else glu(h, t))
        if trace is not None:
            trace.append(x.clone())
    return norm(x, "final.norm") @ w["head"].T * float(config.get("logit_scale", 1.0))


def greedy(config: dict, tensors: Dict[str, torch.Tensor], prompt: List[int], n_new: int) -> List[int]:
    seq = list(prompt)
    for _ in range(n_new):
        seq.append(int(forward(config, tensors, seq)[-1].argmax()))
    return seq[len(prompt):]
