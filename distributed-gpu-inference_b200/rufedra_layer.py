"""Rufedra: a decoder over an fp32 residual stream whose sublayers are normed on the way in AND on the way out,

    x <- x + s1 * N1b(mixer(N1(x)));   x <- x + s2 * N2b(ff(N2(x)));       N an RMS norm, s1 and s2 per-channel layer scales,

with one of two mixers per layer, in any order:

  ``delta``     gated delta rule with one decay per head: q, k and v pass a short causal convolution and SiLU, q and k are made
                unit vectors per head, ``S <- g S; u = beta (v - S^T k); S <- S + k u^T; o = S^T q``; the read-outs are made
                unit-RMS per head, weighted and gated by ``silu(W_g h)``.
  ``parallel``  two mixers side by side on the same input, added with fixed weights ``a_l left + a_r right``:
                left   grouped-query sliding-window attention whose VALUES ARE THE PROJECTED KEYS (before rotation and norm); q
                       and k carry biases, are rotated over their first dimensions (pairs ``(i, i + half)``) and then divided
                       by their RMS per head; every output channel passes a sigmoid gate.
                right  a selective state space: a state per channel, ``S <- e^(dt A) S + dt x B``, ``y = S.C + D x``, with step
                       sizes from a low-rank projection, behind a short convolution with bias and SiLU, gated by ``silu(z)``.

Feed-forward (some layers have none): ``W_down (gelu_tanh(W_gate h) * (W_up h))``.

A ``delta`` layer keeps a state slot per live sequence (matrices and the convolutions' last inputs), a ``parallel`` layer pages AND
a state slot.  One GEMM produces every projection a mixer takes from its input; both sides of a parallel layer write their outputs
side by side into one buffer and one GEMM over the two output projections placed side by side adds them.  The branch weights ride
along: ``N(a_l L + a_r R) = sign(a_l) N'(L + (a_r / a_l) R)`` with N' using ``eps / a_l^2``, so ``a_r / a_l`` scales the right
branch's fp32 outputs before they are rounded and nothing else changes.  Every residual update also forms the next sublayer's
normed input.

The modules follow the calling convention of ``ModelShard.forward`` (reference:
worker/distributed/model_shard.py:205-215): ``layer(h, attention_mask=, position_ids=, past_key_value=, use_cache=)
-> (h, present)`` with ``h`` the packed fp32 residual ``[n_tok, width]`` of one step and ``past_key_value`` a
``RaggedLayerCache``.  Matrix products are torch GEMMs; everything between them is a kernel of ``mixer_ops``.  There is no
dense / CPU mode.

Checkpoint names: ``embed``, ``l<i>.norm1|norm1b|norm2|norm2b|ls1|ls2``, ``l<i>.mix.*`` (``mix.left.*``, ``mix.right.*``),
``l<i>.mlp.*``, ``final.norm``, ``head``; linear weights are ``[out, in]``.
"""
from __future__ import annotations

import math
from typing import Any, Dict, List, Optional, Sequence, Tuple

import torch
import torch.nn as nn
import torch.nn.functional as F

from . import mixer_ops
from .fibirax_layer import wavelength_scaled_frequencies
from .paged_layer import RaggedLayerCache
from .petipel_layer import _param
from .sanesun_layer import UNIT_NORM_EPS, PlainRMSNorm, ScaledFloatEmbedding, _pad8
from .vatazen_layer import LatentRotaryAttention
from .worker.distributed.model_shard import ModelShard
from .zuderax_layer import ScaledHead, _fused

MIXERS = ("delta", "parallel")


class RufedraConfig:
    """``config.json`` of the design, plus the attribute names the rest of the framework reads from a config."""

    def __init__(self, raw: Dict[str, Any]):
        self.raw = raw
        self.architecture = raw.get("architecture", "Rufedra")
        self.layers: List[Dict[str, Any]] = list(raw["layers"])
        self.width = int(raw["width"])
        self.vocab = int(raw["vocab"])
        self.eps = float(raw["norm"]["eps"])
        self.embed_scale = float((raw.get("embedding") or {}).get("scale", 1.0))
        self.logit_scale = float(raw.get("logit_scale", 1.0))
        for i, layer in enumerate(self.layers):
            if layer["type"] not in MIXERS:
                raise NotImplementedError(f"layer {i}: unknown mixer type {layer['type']!r}")
            m = layer["mixer"] if layer["type"] == "delta" else layer["mixer"]["left"]
            if int(m["heads"]) % int(m.get("kv_heads", m["heads"])):
                raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
            if layer["type"] == "parallel":
                dims = int((m.get("rot") or {}).get("dims", 0))
                if dims % 2 or dims > int(m["dim"]):
                    raise ValueError(f"layer {i}: rot.dims must be even and at most dim")
                if int(m.get("vdim", m["dim"])) != int(m["dim"]):
                    raise ValueError(f"layer {i}: values that are the keys have the keys' size")
            mlp = layer.get("mlp")
            if mlp is not None and mlp.get("kind", "dense") != "dense":
                raise NotImplementedError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
        # names shared with the other model classes
        self.hidden_size = self.width
        self.vocab_size = self.vocab
        self.num_hidden_layers = len(self.layers)
        self.num_attention_heads = max(int(l["mixer"].get("left", l["mixer"])["heads"]) for l in self.layers)

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "RufedraConfig":
        return cls(raw)

    def kv_shape(self, i: int) -> Optional[Tuple[int, int, int]]:
        if self.layers[i]["type"] != "parallel":
            return None
        m = self.layers[i]["mixer"]["left"]
        return int(m.get("kv_heads", m["heads"])), int(m["dim"]), int(m["dim"])

    def state_shape(self, i: int):
        """Per live sequence: the state and the convolutions' last ``taps - 1`` inputs (q | k | v, or x)."""
        m = self.layers[i]["mixer"]
        if self.layers[i]["type"] == "delta":
            H, G, dk, dv = int(m["heads"]), int(m.get("kv_heads", m["heads"])), int(m["dim"]), int(m["vdim"])
            return [(H, dk, dv), (int(m["conv"]) - 1, 2 * G * dk + H * dv)]
        m = m["right"]
        return [(int(m["inner"]), int(m["state"])), (int(m["conv"]) - 1, int(m["inner"]))]


class HeadDeltaMixer(nn.Module):
    """The ``delta`` mixer.  Launches per step: the input GEMM (q | k | v | output gate | b | a), convolution + SiLU of q, k and v,
    the delta rule (unit norms, decays and write strengths formed inside), the gated read-out norm, the output GEMM."""

    norm_sign = 1.0

    def __init__(self, spec: Dict[str, Any], t: Dict[str, torch.Tensor], eps: float, device, dtype):
        super().__init__()
        self.H, self.G = int(spec["heads"]), int(spec.get("kv_heads", spec["heads"]))
        self.dk, self.dv = int(spec["dim"]), int(spec["vdim"])
        self.eps = self.norm_eps = eps
        self.n_conv = 2 * self.G * self.dk + self.H * self.dv
        self.w_in, self.cuts = _fused([torch.cat([t["q"], t["k"], t["v"]], dim=0), t["g"], t["b"], t["a"]], device, dtype)
        self.w_conv = _param(torch.cat([t["q.conv"], t["k.conv"], t["v.conv"]], dim=0), device, dtype)
        if self.w_conv.shape != (self.n_conv, int(spec["conv"])):
            raise ValueError("the convolutions hold one row of taps per q, k and v channel")
        self.dt_bias, self.a_log = _param(t["dt_bias"], device, dtype), _param(t["A_log"], device, dtype)
        self.norm_w = _param(t["norm"], device, dtype)
        self.w_o = _param(t["o"], device, dtype)

    def forward(self, h: torch.Tensor, cache: RaggedLayerCache) -> torch.Tensor:
        st, c, H, G, dk, dv = cache.state, self.cuts, self.H, self.G, self.dk, self.dv
        state, tail = cache.rstate
        proj = F.linear(h, self.w_in)
        qkv = mixer_ops.causal_conv_silu(proj[:, :self.n_conv], self.w_conv, tail, st.scan_seqs, st.max_count())
        o = mixer_ops.delta_scan(qkv[:, :G * dk], qkv[:, G * dk:2 * G * dk], qkv[:, 2 * G * dk:], proj[:, c[2]:c[2] + H],
                                 proj[:, c[3]:c[3] + H], self.dt_bias, self.a_log, state, st.scan_seqs, G, UNIT_NORM_EPS,
                                 dk ** -0.5, max_count=st.max_count())
        y = mixer_ops.head_norm_act_gate(o, self.norm_w, proj[:, c[1]:c[1] + H * dv], self.eps, h.dtype, gate_act="silu")
        return F.linear(y, self.w_o)


class KeyValueSelectiveMixer(nn.Module):
    """The ``parallel`` mixer.  Launches per step: the input GEMM (left q | k | gate, right x | z), rotation + norm + append,
    attention with its gate, convolution + SiLU, the GEMMs of step sizes, B and C, the selective scan with its gate, the output
    GEMM."""

    def __init__(self, spec: Dict[str, Any], t: Dict[str, torch.Tensor], eps: float, device, dtype):
        super().__init__()
        left, right = spec["left"], spec["right"]
        lt = {k[5:]: v for k, v in t.items() if k.startswith("left.")}
        rt = {k[6:]: v for k, v in t.items() if k.startswith("right.")}
        self.eps = eps
        # left
        self.H, self.G, self.dk = int(left["heads"]), int(left.get("kv_heads", left["heads"])), int(left["dim"])
        self.scale = float(left["scale"])
        self.window = int((left.get("mask") or {}).get("size", 0))
        rot = left.get("rot") or {}
        freqs = wavelength_scaled_frequencies(int(rot.get("dims", 0)), float(rot.get("base", 10000.0)), None)
        self.register_buffer("freqs", freqs.to(device) if freqs.numel() else None, persistent=False)
        # right
        self.inner, self.N, self.rank = int(right["inner"]), int(right["state"]), int(right["dt_rank"])
        if rt["in"].shape[0] != 2 * self.inner or rt["x"].shape[0] != self.rank + 2 * self.N:
            raise ValueError("the right side projects to x | z, and x to step sizes | B | C")
        sections = [lt["q"], lt["k"], lt["g"], rt["in"][:self.inner], rt["in"][self.inner:]]
        self.w_in, self.cuts = _fused(sections, device, dtype)
        bias = [lt["q.b"], lt["k.b"]] + [torch.zeros(s.shape[0], dtype=s.dtype) for s in sections[2:]]
        self.b_in = _param(torch.cat([_pad8(b) for b in bias], dim=0), device, dtype)
        self.w_conv, self.b_conv = _param(rt["conv"], device, dtype), _param(rt["conv.b"], device, dtype)
        self.w_x, self.x_cuts = _fused([rt["x"][:self.rank], rt["x"][self.rank:self.rank + self.N], rt["x"][self.rank + self.N:]],
                                       device, dtype)
        self.w_dt = _param(rt["dt"], device, dtype)
        f32 = lambda name: _param(rt[name], device, torch.float32)  # noqa: E731
        self.dt_bias, self.skip = f32("dt.b"), f32("D")
        self.rates = _param(-torch.exp(rt["A_log"].to(torch.float64)), device, torch.float32)
        # the two output projections side by side; the branch weights are folded as the module docstring says
        a_l, a_r = float(spec["left_scale"]), float(spec["right_scale"])
        c = a_l if a_l != 0.0 else 1.0
        self.right_gain = a_r / c
        self.norm_sign, self.norm_eps = (1.0 if c > 0 else -1.0), eps / (c * c)
        self.Kl = self.H * self.dk
        self.right_at = self.Kl + (-self.Kl % 8)
        w_ol = lt["o"] if a_l != 0.0 else torch.zeros_like(lt["o"])
        w_out = torch.cat([_pad8(w_ol.t()), _pad8(rt["o"].t())], dim=0).t()
        self.gaps = [(self.Kl, self.right_at), (self.right_at + self.inner, w_out.shape[1])]
        self.w_out = _param(w_out, device, dtype)
        self.tensor_cores = mixer_ops.mixed_prompt_attention_supported(self.H, self.G, self.dk, self.dk, False, False, False,
                                                                       self.w_in.dtype)
        self.rows = (self.tensor_cores and self.G == 1 and self.H >= LatentRotaryAttention.HEADS_AS_ROWS_FROM and
                     mixer_ops.heads_as_rows_supported(self.H, self.dk, self.dk, self.w_in.dtype))

    def forward(self, h: torch.Tensor, cache: RaggedLayerCache) -> torch.Tensor:
        st, n, c = cache.state, h.shape[0], self.cuts
        H, G, dk, inner, N, x_cuts = self.H, self.G, self.dk, self.inner, self.N, self.x_cuts
        state, tail = cache.rstate
        proj = F.linear(h, self.w_in, self.b_in)
        buf = torch.empty((n, self.w_out.shape[1]), dtype=h.dtype, device=h.device)
        for lo, hi in self.gaps:
            if hi > lo:
                buf[:, lo:hi].zero_()
        # left: attention over the pages; the values are the keys as projected
        q, k, gate = proj[:, :H * dk], proj[:, c[1]:c[1] + G * dk], proj[:, c[2]:c[2] + H * dk]
        mixer_ops.qknorm_rotary_append(q, k, k, None, None, self.eps, self.freqs, cache.k_pool, cache.v_pool, st.slot_mapping,
                                       st.tok_pos, H, interleaved=False, unit_norm=True)
        attn = buf[:, :self.Kl].unflatten(1, (H, dk))
        if self.tensor_cores:
            tiles, _ = st.prompt_tiles(1, mixer_ops.PROMPT_TILE_TOKENS)
            mixer_ops.mixed_prompt_attention(attn, q.unflatten(1, (H, dk)), cache.k_pool, cache.v_pool, st.block_tables, tiles,
                                             st.tok_pos, self.scale, window=self.window, gate=gate,
                                             max_context=st.max_context(), heads_as_rows=self.rows and st.max_count() == 1)
        else:
            mixer_ops.mixed_paged_attention(attn, q.unflatten(1, (H, dk)), cache.k_pool, cache.v_pool, st.block_tables,
                                            st.tok_row, st.tok_pos, self.scale, window=self.window, gate=gate)
        # right: the selective scan over the state slots
        x = mixer_ops.causal_conv_silu(proj[:, c[3]:c[3] + inner], self.w_conv, tail, st.scan_seqs, st.max_count(),
                                       bias=self.b_conv)
        p = F.linear(x, self.w_x)
        dt = F.linear(p[:, :self.rank], self.w_dt)
        mixer_ops.selective_scan(x, dt, p[:, x_cuts[1]:x_cuts[1] + N], p[:, x_cuts[2]:x_cuts[2] + N],
                                 proj[:, c[4]:c[4] + inner], self.dt_bias, self.rates, self.skip, state, st.scan_seqs,
                                 gain=self.right_gain, out=buf[:, self.right_at:self.right_at + inner],
                                 max_count=st.max_count())
        return F.linear(buf, self.w_out)


class GeluGLU(nn.Module):
    """``W_down (gelu_tanh(W_gate h) * (W_up h))``."""

    def __init__(self, t: Dict[str, torch.Tensor], device, dtype):
        super().__init__()
        self.w_gu = _param(torch.cat([t["gate"], t["up"]], dim=0), device, dtype)
        self.w_down = _param(t["down"], device, dtype)

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return F.linear(mixer_ops.gelu_glu(F.linear(h, self.w_gu)), self.w_down)


class RufedraDecoderLayer(nn.Module):
    """One layer; see the module docstring.  ``next_norm_weight`` (set by the builder when another layer of the same shard
    follows) lets the layer's last residual update also form that layer's normed input."""

    def __init__(self, config: RufedraConfig, layer_idx: int, t: Dict[str, torch.Tensor], device=None, dtype=None):
        super().__init__()
        spec = config.layers[layer_idx]
        self.layer_idx, self.kind, self.eps = layer_idx, spec["type"], config.eps
        mix = {k[4:]: v for k, v in t.items() if k.startswith("mix.")}
        cls = HeadDeltaMixer if self.kind == "delta" else KeyValueSelectiveMixer
        self.mixer = cls(spec["mixer"], mix, self.eps, device, dtype)
        self.norm1 = PlainRMSNorm(config.width, self.eps, device, dtype)
        with torch.no_grad():
            self.norm1.weight.copy_(t["norm1"])
        self.norm1b, self.ls1 = _param(t["norm1b"], device, dtype), _param(t["ls1"], device, dtype)
        self.mlp = None
        if spec.get("mlp") is not None:
            self.mlp = GeluGLU({k[4:]: v for k, v in t.items() if k.startswith("mlp.")}, device, dtype)
            self.norm2 = _param(t["norm2"], device, dtype)
            self.norm2b, self.ls2 = _param(t["norm2b"], device, dtype), _param(t["ls2"], device, dtype)
        self.next_norm_weight: Optional[torch.Tensor] = None

    def forward(self, hidden_states: torch.Tensor, attention_mask=None, position_ids=None,
                past_key_value: Optional[RaggedLayerCache] = None, use_cache: bool = True):
        if not isinstance(past_key_value, RaggedLayerCache):
            raise TypeError("RufedraDecoderLayer needs a RaggedLayerCache handle in past_key_value")
        x, st = hidden_states, past_key_value.state
        if x.dtype != torch.float32 or x.dim() != 2:
            raise TypeError("the residual stream is a packed fp32 [n_tok, width] tensor")
        h = st.pending_norm if st.pending_norm is not None else self.norm1(x)
        y = self.mixer(h, past_key_value)
        w_next = self.norm2 if self.mlp is not None else self.next_norm_weight
        h = mixer_ops.sandwich_residual(x, y, self.norm1b, self.ls1, self.mixer.norm_eps, w_next, self.eps,
                                        sign=self.mixer.norm_sign)
        if self.mlp is not None:
            h = mixer_ops.sandwich_residual(x, self.mlp(h), self.norm2b, self.ls2, self.eps, self.next_norm_weight, self.eps)
        st.pending_norm = h
        return x, (past_key_value if use_cache else None)


def build_shards(config: RufedraConfig, tensors: Dict[str, torch.Tensor], ranges: Sequence[Tuple[int, int]],
                 device: str, dtype: torch.dtype) -> List[ModelShard]:
    """``ModelShard``s for layer ranges holding the weights of a checkpoint's name -> tensor dict."""
    shards = []
    total = config.num_hidden_layers
    for start, end in ranges:
        layers = []
        for i in range(start, end):
            pre = f"l{i}."
            layers.append(RufedraDecoderLayer(config, i, {k[len(pre):]: v for k, v in tensors.items() if k.startswith(pre)},
                                              device, dtype))
        for a, b in zip(layers[:-1], layers[1:]):
            a.next_norm_weight = b.norm1.weight
        embed = norm = head = None
        if start == 0:
            embed = ScaledFloatEmbedding(config.vocab, config.width, device=device, dtype=dtype, scale=config.embed_scale)
            embed.weight.requires_grad_(False)
            with torch.no_grad():
                embed.weight.copy_(tensors["embed"])
        if end == total:
            norm = PlainRMSNorm(config.width, config.eps, device, dtype)
            head = ScaledHead(config.width, config.vocab, bias=False, device=device, dtype=dtype)
            head.logit_scale = config.logit_scale
            head.weight.requires_grad_(False)
            with torch.no_grad():
                norm.weight.copy_(tensors["final.norm"])
                head.weight.copy_(tensors["head"])
        shards.append(ModelShard.from_layers(config, layers, start, end, device, dtype, embed, norm, head,
                                             model_id="rufedra").eval())
    return shards


def random_checkpoint(config: RufedraConfig, seed: int = 0, dtype: torch.dtype = torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random weights with the checkpoint's names and shapes (for tests and benchmarks; not a trained model).
    Projections ~ N(0, gain / fan_in); norms, layer scales, decays and step sizes are chosen so that every term of the design
    contributes."""
    g = torch.Generator().manual_seed(seed)
    W = config.width

    def lin(out, inp, gain=1.0):
        return (torch.randn(out, inp, generator=g) * gain / math.sqrt(inp)).to(dtype)

    def vec(n, s=1.0, mean=0.0):
        return (mean + s * torch.randn(n, generator=g)).to(dtype)

    def conv(rows, taps):
        return (torch.randn(rows, taps, generator=g) / math.sqrt(taps)).to(dtype)

    t: Dict[str, torch.Tensor] = {"embed": (torch.randn(config.vocab, W, generator=g) / config.embed_scale).to(dtype)}
    for i, layer in enumerate(config.layers):
        pre, m = f"l{i}.mix.", layer["mixer"]
        for name in ("norm1", "norm1b"):
            t[f"l{i}.{name}"] = vec(W, 0.2, 1.0)
        t[f"l{i}.ls1"] = vec(W, 0.15, 0.6)
        if layer["type"] == "delta":
            H, G, dk, dv = int(m["heads"]), int(m.get("kv_heads", m["heads"])), int(m["dim"]), int(m["vdim"])
            for name, rows in (("q", G * dk), ("k", G * dk), ("v", H * dv)):
                t[pre + name], t[pre + name + ".conv"] = lin(rows, W, 1.5), conv(rows, int(m["conv"]))
            t[pre + "b"], t[pre + "a"], t[pre + "g"] = lin(H, W, 1.5), lin(H, W, 1.5), lin(H * dv, W, 1.5)
            t[pre + "A_log"], t[pre + "dt_bias"] = vec(H, 0.8, -0.5), vec(H, 0.8, -2.0)
            t[pre + "norm"], t[pre + "o"] = vec(dv, 0.2, 1.0), lin(W, H * dv)
        else:
            left, right = m["left"], m["right"]
            H, G, dk = int(left["heads"]), int(left.get("kv_heads", left["heads"])), int(left["dim"])
            for name, rows in (("q", H * dk), ("k", G * dk)):
                t[pre + "left." + name], t[pre + "left." + name + ".b"] = lin(rows, W, 1.0), vec(rows, 0.4)
            t[pre + "left.g"], t[pre + "left.o"] = lin(H * dk, W, 1.5), lin(W, H * dk, 1.5)
            I, N, r = int(right["inner"]), int(right["state"]), int(right["dt_rank"])
            t[pre + "right.in"] = lin(2 * I, W, 1.5)
            t[pre + "right.conv"], t[pre + "right.conv.b"] = conv(I, int(right["conv"])), vec(I, 0.2)
            t[pre + "right.x"] = lin(r + 2 * N, I, 2.0)
            t[pre + "right.dt"], t[pre + "right.dt.b"] = lin(I, r), vec(I, 1.0, -2.5)
            t[pre + "right.A_log"] = (torch.log(torch.arange(1, N + 1, dtype=torch.float32)).repeat(I, 1)
                                      + 0.3 * torch.randn(I, N, generator=g)).to(dtype)
            t[pre + "right.D"], t[pre + "right.o"] = vec(I, 0.3, 0.5), lin(W, I)
        if layer.get("mlp") is None:
            continue
        for name in ("norm2", "norm2b"):
            t[f"l{i}.{name}"] = vec(W, 0.2, 1.0)
        t[f"l{i}.ls2"] = vec(W, 0.15, 0.6)
        ff = int(layer["mlp"]["ff"])
        t[f"l{i}.mlp.gate"], t[f"l{i}.mlp.up"], t[f"l{i}.mlp.down"] = lin(ff, W, 1.5), lin(ff, W, 1.5), lin(W, ff)
    t["final.norm"] = vec(W, 0.2, 1.0)
    t["head"] = lin(config.vocab, W)
    return t
