"""Zuderax: a pre-norm decoder over an fp32 residual stream,

    x <- x + mixer(D1(x));   x <- x + ff(D2(x));       D(x) = tanh(alpha x) * w + b   (no statistic),

with one of three mixers per layer, in any order:

  ``latent_attention``  sliding-window softmax attention whose keys and values are up-projections of one normed latent row
                        per token plus one rotated key part shared by all heads (rotary pairs ``(i, i + half)``); served in
                        the absorbed form over a one-head pool, the mixer class Vatazen's latent layers use.
  ``mlstm``             a matrix memory ``S <- e^(f + m' - m) S + e^(i - m) k v^T`` per head with soft-capped log gates and a
                        running maximum ``m`` that starts at 0, a normaliser ``n`` of the same recurrence, read out as
                        ``S^T q / (max(|n.q|, e^-m) + 1e-6)``, made unit-RMS per head and gated by a sigmoid.
  ``mamba2``            a state ``S <- e^(-e^A dt) S + dt B x^T`` per head with B and C shared by groups of heads, ``y = S^T C +
                        D x``; x, B and C pass a short causal convolution with bias and SiLU; ``y * silu(z)`` is normed in
                        equal parts of the row.

Both recurrences decay a matrix per head by ONE number per token, so they share the scan and the single-token kernel and
differ in where the decay comes from and in how the read-out is normed.  Their fp32 states (matrix, normaliser and maximum;
matrix and the convolution's last inputs) live in the slot pool per live sequence; latent layers keep pages.

Feed-forward: ``W_down (silu(W_gate h) * (W_up h))``, or a mixture of such experts: sigmoid scores, choice by score + a
correction inside the expert groups whose two best choice scores have the largest sum, weights = scores times a constant
(not renormalised), plus a shared expert weighted by a sigmoid per token.  The shared expert's gate is one more output of
the router's launch; the weighted combine, the residual update and the next sublayer's norm are one launch.

A layer with ``weights_of: j`` runs layer j's weights (the same module) with pages or a state of its own.

The modules follow the calling convention of ``ModelShard.forward`` (reference:
worker/distributed/model_shard.py:205-215): ``layer(h, attention_mask=, position_ids=, past_key_value=, use_cache=)
-> (h, present)`` with ``h`` the packed fp32 residual ``[n_tok, width]`` of one step and ``past_key_value`` a
``RaggedLayerCache``.  Matrix products are torch GEMMs; everything between them is a kernel of ``mixer_ops``.  There is no
dense / CPU mode.

Checkpoint names: ``embed``, ``l<i>.norm1|norm2`` with ``.alpha`` and ``.b``, ``l<i>.mix.*``, ``l<i>.mlp.*``, ``final.norm``,
``head``; linear weights are ``[out, in]``.
"""
from __future__ import annotations

import math
from typing import Any, Dict, List, Optional, Sequence, Tuple

import torch
import torch.nn as nn
import torch.nn.functional as F

from . import mixer_ops
from .fibirax_layer import GroupedSoftmaxMoE
from .paged_layer import RaggedLayerCache
from .petipel_layer import FloatEmbedding, _param
from .sanesun_layer import _pad8
from .vatazen_layer import LatentRotaryAttention
from .worker.distributed.model_shard import ModelShard

MIXERS = ("latent_attention", "mlstm", "mamba2")
READOUT_FLOOR = 1e-6       # added to the matrix memory's read-out denominator; fixed by the design


class ZuderaxConfig:
    """``config.json`` of the design, plus the attribute names the rest of the framework reads from a config."""

    def __init__(self, raw: Dict[str, Any]):
        self.raw = raw
        self.architecture = raw.get("architecture", "Zuderax")
        self.layers: List[Dict[str, Any]] = list(raw["layers"])
        self.width = int(raw["width"])
        self.vocab = int(raw["vocab"])
        self.eps = float(raw["norm"]["eps"])
        self.logit_scale = float(raw.get("logit_scale", 1.0))
        for i, layer in enumerate(self.layers):
            if layer["type"] not in MIXERS:
                raise NotImplementedError(f"layer {i}: unknown mixer type {layer['type']!r}")
            m = layer["mixer"]
            if layer["type"] == "latent_attention":
                dims = int((m.get("rot") or {}).get("dims", 0))
                if dims > int(m["rot_dim"]) or dims % 2:
                    raise ValueError(f"layer {i}: rot.dims must be even and at most rot_dim")
            if layer["type"] == "mamba2":
                H, dv = int(m["heads"]), int(m["vdim"])
                if H % int(m["groups"]) or (H * dv) % int(m.get("norm_groups", 1)):
                    raise ValueError(f"layer {i}: groups must divide the heads and norm_groups the inner size")
            src = layer.get("weights_of")
            if src is not None:
                if not 0 <= int(src) < len(self.layers) or self.layers[int(src)]["type"] != layer["type"]:
                    raise ValueError(f"layer {i}: weights_of {src} names no layer of the same kind")
                self.source(i)      # raises when the references run in a circle
            mlp = layer.get("mlp")
            if mlp is None:
                continue
            if mlp.get("kind", "dense") not in ("dense", "moe"):
                raise NotImplementedError(f"layer {i}: unknown feed-forward kind {mlp['kind']!r}")
            if mlp.get("kind") == "moe" and int(mlp["router"]["experts"]) % int((mlp["router"].get("groups") or {}).get("count", 1)):
                raise ValueError(f"layer {i}: experts do not divide into groups")
        # names shared with the other model classes
        self.hidden_size = self.width
        self.vocab_size = self.vocab
        self.num_hidden_layers = len(self.layers)
        self.num_attention_heads = max(int(l["mixer"]["heads"]) for l in self.layers)

    @classmethod
    def from_dict(cls, raw: Dict[str, Any]) -> "ZuderaxConfig":
        return cls(raw)

    def source(self, i: int) -> int:
        """The layer whose tensors layer ``i`` runs (itself unless it names another)."""
        for _ in range(len(self.layers) + 1):
            src = self.layers[i].get("weights_of")
            if src is None:
                return i
            i = int(src)
        raise ValueError("weights_of runs in a circle")

    def kv_shape(self, i: int) -> Optional[Tuple[int, int, int]]:
        """A latent layer keeps one row ``[latent | rotated key part]`` per token and no value pool."""
        m = self.layers[i]["mixer"]
        if self.layers[i]["type"] != "latent_attention":
            return None
        return 1, int(m["kv_rank"]) + int(m["rot_dim"]), 0

    def state_shape(self, i: int):
        """Per live sequence: matrix, normaliser and running maximum of a matrix memory; matrix and the convolution's last
        ``taps - 1`` inputs (x | B | C) of a state space layer."""
        kind, m = self.layers[i]["type"], self.layers[i]["mixer"]
        H, dv = int(m["heads"]), int(m["vdim"])
        if kind == "mlstm":
            return [(H, int(m["dim"]), dv), (H, int(m["dim"])), (H,)]
        if kind == "mamba2":
            N = int(m["state"])
            return [(H, N, dv), (int(m["conv"]) - 1, H * dv + 2 * int(m["groups"]) * N)]
        return None


class DynTanhNorm(nn.Module):
    """``tanh(alpha x) * weight + bias`` over fp32 rows; the weight's dtype out."""

    def __init__(self, t: Dict[str, torch.Tensor], name: str, device=None, dtype=None):
        super().__init__()
        self.weight, self.bias = _param(t[name], device, dtype), _param(t[name + ".b"], device, dtype)
        self.alpha = float(t[name + ".alpha"])

    def args(self):
        return self.weight, self.bias, self.alpha

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        return mixer_ops.residual_dyn_tanh(x, None, self.args())


class ScaledHead(nn.Linear):
    """An output head whose logits carry a constant factor."""

    logit_scale = 1.0

    def forward(self, x: torch.Tensor) -> torch.Tensor:
        y = super().forward(x)
        return y if self.logit_scale == 1.0 else y * self.logit_scale


def _fused(sections: Sequence[torch.Tensor], device, dtype):
    """One ``[out, in]`` weight from several (each padded to 8 rows) and where each section starts."""
    cuts = [0]
    for s in sections:
        cuts.append(cuts[-1] + s.shape[0] + (-s.shape[0] % 8))
    return _param(torch.cat([_pad8(s) for s in sections], dim=0), device, dtype), cuts


class MatrixMemoryMixer(nn.Module):
    """The ``mlstm`` mixer.  Launches per step: the input GEMM (q | k | v | output gate | i | f), the gates' scan, the state
    scan, the read-out norm, the output GEMM; a step of single tokens forms the gates inside the state launch."""

    def __init__(self, spec: Dict[str, Any], t: Dict[str, torch.Tensor], eps: float, device, dtype):
        super().__init__()
        self.H, self.dk, self.dv = int(spec["heads"]), int(spec["dim"]), int(spec["vdim"])
        self.cap, self.eps = float(spec["gate_cap"]), eps
        self.w_in, self.cuts = _fused([t["q"], t["k"], t["v"], t["g"], t["i"], t["f"]], device, dtype)
        self.b_i, self.b_f = _param(t["i.b"], device, torch.float32), _param(t["f.b"], device, torch.float32)
        self.norm_w = _param(t["norm"], device, dtype)
        self.w_o = _param(t["o"], device, dtype)

    def forward(self, h: torch.Tensor, cache: RaggedLayerCache) -> torch.Tensor:
        st, c, H, dk, dv = cache.state, self.cuts, self.H, self.dk, self.dv
        S, n_state, m_state = cache.rstate
        proj = F.linear(h, self.w_in)
        q, k, v = proj[:, :H * dk], proj[:, c[1]:c[1] + H * dk], proj[:, c[2]:c[2] + H * dv]
        gate, zi, zf = proj[:, c[3]:c[3] + H * dv], proj[:, c[4]:c[4] + H], proj[:, c[5]:c[5] + H]
        if st.max_count() == 1:
            o, nq, m = mixer_ops.decay_step(q, k, v, ("capped", zi, zf, self.b_i, self.b_f, self.cap), S, st.scan_seqs, H,
                                            q_scale=dk ** -0.5, nstate=n_state, m_state=m_state)
            y = mixer_ops.normalized_head_out(o, nq, m, READOUT_FLOOR, self.norm_w, gate, self.eps, m_state, st.scan_seqs)
        else:
            log_decay, coef, m = mixer_ops.capped_gates(zi, zf, self.b_i, self.b_f, self.cap, m_state, st.scan_seqs)
            o, nq = mixer_ops.decay_scan(q, k, v, log_decay, coef, S, st.scan_seqs, H, q_scale=dk ** -0.5, nstate=n_state,
                                         max_count=st.max_count())
            y = mixer_ops.normalized_head_out(o, nq, m, READOUT_FLOOR, self.norm_w, gate, self.eps)
        return F.linear(y, self.w_o)


class StateSpaceMixer(nn.Module):
    """The ``mamba2`` mixer.  Launches per step: the input GEMM (z | x | B | C | dt), convolution + SiLU of x, B and C, the
    step sizes, the state scan, the gated norm, the output GEMM; a step of single tokens forms the step sizes inside the
    state launch."""

    def __init__(self, spec: Dict[str, Any], t: Dict[str, torch.Tensor], eps: float, device, dtype):
        super().__init__()
        self.H, self.dv, self.N, self.G = int(spec["heads"]), int(spec["vdim"]), int(spec["state"]), int(spec["groups"])
        self.parts, self.eps = int(spec.get("norm_groups", 1)), eps
        self.inner = self.H * self.dv
        n_conv = self.inner + 2 * self.G * self.N
        if t["in"].shape[0] != self.inner + n_conv + self.H or t["conv"].shape[0] != n_conv:
            raise ValueError("the input projection holds z | x | B | C | dt")
        self.n_conv = n_conv
        self.w_in, self.cuts = _fused([t["in"][:self.inner], t["in"][self.inner:self.inner + n_conv],
                                       t["in"][self.inner + n_conv:]], device, dtype)
        self.w_conv = _param(t["conv"], device, dtype)
        self.b_conv = _param(t["conv.b"], device, dtype) if "conv.b" in t else None
        f32 = lambda name: _param(t[name], device, torch.float32)  # noqa: E731
        self.dt_bias, self.a_log, self.skip = f32("dt_bias"), f32("A_log"), f32("D")
        self.norm_w = _param(t["norm"], device, dtype)
        self.w_o = _param(t["o"], device, dtype)

    def forward(self, h: torch.Tensor, cache: RaggedLayerCache) -> torch.Tensor:
        st, c, G, N = cache.state, self.cuts, self.G, self.N
        S, tail = cache.rstate
        proj = F.linear(h, self.w_in)
        xbc = mixer_ops.causal_conv_silu(proj[:, c[1]:c[1] + self.n_conv], self.w_conv, tail, st.scan_seqs, st.max_count(),
                                         bias=self.b_conv)
        x = xbc[:, :self.inner]
        B, C = xbc[:, self.inner:self.inner + G * N], xbc[:, self.inner + G * N:]
        dt = proj[:, c[2]:c[2] + self.H]
        if st.max_count() == 1:
            y, _, _ = mixer_ops.decay_step(C, B, x, ("step", dt, self.dt_bias, self.a_log), S, st.scan_seqs, G, skip=self.skip)
        else:
            log_decay, coef = mixer_ops.step_sizes(dt, self.dt_bias, self.a_log)
            y, _ = mixer_ops.decay_scan(C, B, x, log_decay, coef, S, st.scan_seqs, G, skip=self.skip,
                                        max_count=st.max_count())
        return F.linear(mixer_ops.gated_part_norm(y, proj[:, :self.inner], self.norm_w, self.eps, self.parts), self.w_o)


class SiluGLU(nn.Module):
    """``W_down (silu(W_gate h) * (W_up h))``."""

    def __init__(self, t: Dict[str, torch.Tensor], device, dtype, pre: str = ""):
        super().__init__()
        self.w_gu = _param(torch.cat([t[pre + "gate"], t[pre + "up"]], dim=0), device, dtype)
        self.w_down = _param(t[pre + "down"], device, dtype)

    def forward(self, h: torch.Tensor) -> torch.Tensor:
        return F.linear(mixer_ops.silu_glu(F.linear(h, self.w_gu)), self.w_down)


class SigmoidGroupMoE(GroupedSoftmaxMoE):
    """Experts ``W_down (silu(W_gate h) * (W_up h))`` under the dispatch of ``GroupedSoftmaxMoE``, chosen and weighted by
    sigmoid scores; a shared expert behind a sigmoid per token.  The combine also updates the residual and forms the next
    sublayer's normed input."""

    def __init__(self, spec: Dict[str, Any], t: Dict[str, torch.Tensor], device, dtype):
        nn.Module.__init__(self)
        r = spec["router"]
        self.E, self.ident, self.top = int(r["experts"]), 0, int(r["top"])
        groups = r.get("groups") or {}
        self.groups = int(groups.get("count", 1))
        self.keep = int(groups.get("keep", self.groups))
        self.weight_scale = float(r.get("scale", 1.0))
        if t["router"].shape[0] != self.E:
            raise ValueError("the router has one output per expert")
        self.shared = SiluGLU(t, device, dtype, "shared.") if spec.get("shared") else None
        self.shared_gated = self.shared is not None and "shared.sg" in t
        rows = [t["router"], t["shared.sg"]] if self.shared_gated else [t["router"]]
        self.w_router = _param(torch.cat(rows, dim=0), device, torch.float32)     # the shared gate rides as one more output
        self.correction = _param(t["correction"], device, torch.float32) if "correction" in t else None
        self.w_gu = _param(torch.stack([torch.cat([t[f"e{e}.gate"], t[f"e{e}.up"]], dim=0) for e in range(self.E)]),
                           device, dtype)                                                           # [E, 2 ff, W]
        self.w_down = _param(torch.stack([t[f"e{e}.down"] for e in range(self.E)]), device, dtype)  # [E, W, ff]
        self.grouped = (mixer_ops.grouped_linear_supported(self.w_gu.shape[2], self.w_gu.dtype)
                        and mixer_ops.grouped_linear_supported(self.w_down.shape[2], self.w_down.dtype))
        self._ar = None

    def _activate(self, z: torch.Tensor) -> torch.Tensor:
        return mixer_ops.silu_glu(z)

    def forward(self, h: torch.Tensor, x: torch.Tensor, norm=None) -> Optional[torch.Tensor]:
        """Adds the sublayer's output to the fp32 residual ``x``; returns the normed next input when ``norm`` is given."""
        logits = mixer_ops.router_logits(h, self.w_router)
        ids, w = mixer_ops.sigmoid_group_topk(logits, self.correction, self.E, self.top, self.groups, self.keep,
                                              self.weight_scale)
        ys, where = self._experts(h, ids)
        shared = self.shared(h) if self.shared is not None else None
        return mixer_ops.expert_combine_dyn_tanh(x, ys, where, w, shared, logits[:, self.E] if self.shared_gated else None, norm)


_MIXER_CLASSES = {
    "latent_attention": lambda *a: LatentRotaryAttention(*a, interleaved=False),
    "mlstm": MatrixMemoryMixer,
    "mamba2": StateSpaceMixer,
}


class ZuderaxDecoderLayer(nn.Module):
    """One layer; see the module docstring.  Every residual update also forms the next sublayer's normed input;
    ``next_norm`` (set by the builder when another layer of the same shard follows) extends that over the layer's end.
    ``twin``: the layer whose weights this one runs, when it lives in the same shard."""

    def __init__(self, config: ZuderaxConfig, layer_idx: int, t: Dict[str, torch.Tensor], device=None, dtype=None,
                 twin: Optional["ZuderaxDecoderLayer"] = None):
        super().__init__()
        spec = config.layers[layer_idx]
        self.layer_idx, self.kind, self.eps = layer_idx, spec["type"], config.eps
        self.next_norm: Optional[tuple] = None
        self.mlp = self.norm2 = None
        if twin is not None:
            self.mixer, self.norm1 = twin.mixer, twin.norm1
            if spec.get("mlp") is not None:
                self.mlp, self.norm2 = twin.mlp, twin.norm2
            return
        mix = {k[4:]: v for k, v in t.items() if k.startswith("mix.")}
        self.mixer = _MIXER_CLASSES[self.kind](spec["mixer"], mix, self.eps, device, dtype)
        self.norm1 = DynTanhNorm(t, "norm1", device, dtype)
        if spec.get("mlp") is not None:
            mlp = {k[4:]: v for k, v in t.items() if k.startswith("mlp.")}
            moe = spec["mlp"].get("kind", "dense") == "moe"
            self.mlp = SigmoidGroupMoE(spec["mlp"], mlp, device, dtype) if moe else SiluGLU(mlp, device, dtype)
            self.norm2 = DynTanhNorm(t, "norm2", device, dtype)

    def forward(self, hidden_states: torch.Tensor, attention_mask=None, position_ids=None,
                past_key_value: Optional[RaggedLayerCache] = None, use_cache: bool = True):
        if not isinstance(past_key_value, RaggedLayerCache):
            raise TypeError("ZuderaxDecoderLayer needs a RaggedLayerCache handle in past_key_value")
        x, st = hidden_states, past_key_value.state
        if x.dtype != torch.float32 or x.dim() != 2:
            raise TypeError("the residual stream is a packed fp32 [n_tok, width] tensor")
        h = st.pending_norm if st.pending_norm is not None else self.norm1(x)
        y = self.mixer(h, past_key_value)
        if self.mlp is None:
            st.pending_norm = mixer_ops.residual_dyn_tanh(x, y, self.next_norm)
        else:
            h = mixer_ops.residual_dyn_tanh(x, y, self.norm2.args())
            if isinstance(self.mlp, SigmoidGroupMoE):
                st.pending_norm = self.mlp(h, x, self.next_norm)
            else:
                st.pending_norm = mixer_ops.residual_dyn_tanh(x, self.mlp(h), self.next_norm)
        return x, (past_key_value if use_cache else None)


def build_shards(config: ZuderaxConfig, tensors: Dict[str, torch.Tensor], ranges: Sequence[Tuple[int, int]],
                 device: str, dtype: torch.dtype) -> List[ModelShard]:
    """``ModelShard``s for layer ranges holding the weights of a checkpoint's name -> tensor dict."""
    shards = []
    total = config.num_hidden_layers
    for start, end in ranges:
        layers: List[ZuderaxDecoderLayer] = []
        by_source: Dict[int, ZuderaxDecoderLayer] = {}
        for i in range(start, end):
            src = config.source(i)
            pre = f"l{src}."
            t = {} if src in by_source else {k[len(pre):]: v for k, v in tensors.items() if k.startswith(pre)}
            layers.append(ZuderaxDecoderLayer(config, i, t, device, dtype, twin=by_source.get(src)))
            by_source.setdefault(src, layers[-1])
        for a, b in zip(layers[:-1], layers[1:]):
            a.next_norm = b.norm1.args()
        embed = norm = head = None
        if start == 0:
            embed = FloatEmbedding(config.vocab, config.width, device=device, dtype=dtype)
            embed.weight.requires_grad_(False)
            with torch.no_grad():
                embed.weight.copy_(tensors["embed"])
        if end == total:
            norm = DynTanhNorm(tensors, "final.norm", device, dtype)
            head = ScaledHead(config.width, config.vocab, bias=False, device=device, dtype=dtype)
            head.logit_scale = config.logit_scale
            head.weight.requires_grad_(False)
            with torch.no_grad():
                head.weight.copy_(tensors["head"])
        shards.append(ModelShard.from_layers(config, layers, start, end, device, dtype, embed, norm, head,
                                             model_id="zuderax").eval())
    return shards


def random_checkpoint(config: ZuderaxConfig, seed: int = 0, dtype: torch.dtype = torch.bfloat16) -> Dict[str, torch.Tensor]:
    """Random weights with the checkpoint's names and shapes (for tests and benchmarks; not a trained model).
    Projections ~ N(0, gain / fan_in); norms, gates, step sizes, decays and corrections are chosen so that every term of
    the design contributes."""
    g = torch.Generator().manual_seed(seed)
    W = config.width

    def lin(out, inp, gain=1.0):
        return (torch.randn(out, inp, generator=g) * gain / math.sqrt(inp)).to(dtype)

    def vec(n, s=1.0, mean=0.0):
        return (mean + s * torch.randn(n, generator=g)).to(dtype)

    t: Dict[str, torch.Tensor] = {"embed": (3.0 * torch.randn(config.vocab, W, generator=g)).to(dtype)}

    def norm(name):
        t[name], t[name + ".b"] = vec(W, 0.2, 1.2), vec(W, 0.1)
        t[name + ".alpha"] = (0.25 + 0.2 * torch.rand((), generator=g)).to(dtype)

    for i, layer in enumerate(config.layers):
        if layer.get("weights_of") is not None:
            continue
        pre, m = f"l{i}.mix.", layer["mixer"]
        H, dv = int(m["heads"]), int(m["vdim"])
        norm(f"l{i}.norm1")
        if layer["type"] == "latent_attention":
            dk, r, dr = int(m["dim"]), int(m["kv_rank"]), int(m["rot_dim"])
            t[pre + "q"] = lin(H * (dk + dr), W, 2.0)
            t[pre + "dkv"], t[pre + "dkv.norm"] = lin(r + dr, W, 2.0), vec(r, 0.1, 1.0)
            t[pre + "uk"], t[pre + "uv"] = lin(H * dk, r, 1.5), lin(H * dv, r)
        elif layer["type"] == "mlstm":
            dk = int(m["dim"])
            t[pre + "q"], t[pre + "k"] = lin(H * dk, W, 1.5), lin(H * dk, W, 1.5)
            t[pre + "v"], t[pre + "g"] = lin(H * dv, W), lin(H * dv, W, 2.0)
            t[pre + "i"], t[pre + "i.b"] = lin(H, W, 2.0), vec(H, 1.0, -1.0)
            t[pre + "f"], t[pre + "f.b"] = lin(H, W, 2.0), vec(H, 1.0, 3.0)
            t[pre + "norm"] = vec(H * dv, 0.2, 1.0)
        else:
            N, G, taps = int(m["state"]), int(m["groups"]), int(m["conv"])
            n_conv = H * dv + 2 * G * N
            t[pre + "in"] = lin(H * dv + n_conv + H, W, 1.5)
            t[pre + "conv"] = (torch.randn(n_conv, taps, generator=g) / math.sqrt(taps)).to(dtype)
            t[pre + "conv.b"] = vec(n_conv, 0.2)
            t[pre + "dt_bias"] = vec(H, 1.0, -2.0)
            t[pre + "A_log"], t[pre + "D"] = vec(H, 0.7), vec(H, 0.5, 1.0)
            t[pre + "norm"] = vec(H * dv, 0.2, 1.0)
        t[pre + "o"] = lin(W, H * dv)
        mlp = layer.get("mlp")
        if mlp is None:
            continue
        norm(f"l{i}.norm2")
        pre = f"l{i}.mlp."

        def glu(name, ff):
            t[name + "gate"], t[name + "up"], t[name + "down"] = lin(ff, W, 1.5), lin(ff, W, 1.5), lin(W, ff)

        if mlp.get("kind", "dense") == "dense":
            glu(pre, int(mlp["ff"]))
        else:
            E = int(mlp["router"]["experts"])
            for e in range(E):
                glu(pre + f"e{e}.", int(mlp["expert"]["ff"]))
            t[pre + "router"], t[pre + "correction"] = lin(E, W, 2.0), vec(E, 0.3)
            if mlp.get("shared"):
                glu(pre + "shared.", int(mlp["shared"]["ff"]))
                t[pre + "shared.sg"] = lin(1, W, 2.0)
    norm("final.norm")
    t["head"] = lin(config.vocab, W, 2.0)
    return t
