"""CPU: configuration, registry, pools and checkpoint layout of the Zuderax model class, and sanity of its oracle."""
import math

import pytest
import torch

import dgi_b200  # noqa: F401
from dgi_b200 import model_registry
from dgi_b200 import zuderax_layer as Z
from oracle import zuderax_ref as R

F64 = torch.float64
LATENT = {"type": "latent_attention", "mlp": {"kind": "dense", "ff": 20},
          "mixer": {"heads": 2, "dim": 6, "rot_dim": 4, "vdim": 10, "kv_rank": 14, "scale": 0.3, "mask": {"size": 7},
                    "rot": {"base": 100.0, "dims": 4}}}
MEMORY = {"type": "mlstm", "mixer": {"heads": 3, "dim": 5, "vdim": 6, "gate_cap": 4.0},
          "mlp": {"kind": "moe", "expert": {"ff": 8}, "shared": {"ff": 10},
                  "router": {"experts": 6, "top": 2, "scale": 1.5, "groups": {"count": 3, "keep": 2}}}}
SPACE = {"type": "mamba2", "mixer": {"heads": 4, "vdim": 3, "state": 5, "groups": 2, "conv": 4, "norm_groups": 3}, "mlp": None}
CFG = {"architecture": "Zuderax", "width": 24, "vocab": 19, "norm": {"eps": 1e-5}, "logit_scale": 0.7,
       "layers": [LATENT, MEMORY, SPACE, dict(MEMORY, weights_of=1)]}


def test_config_names_pools_and_states():
    cfg = Z.ZuderaxConfig.from_dict(CFG)
    assert cfg.num_hidden_layers == 4 and cfg.hidden_size == 24 and cfg.vocab_size == 19 and cfg.logit_scale == 0.7
    assert cfg.kv_shape(0) == (1, 18, 0) and cfg.state_shape(0) is None          # one row [latent | rotated key part] per token
    assert cfg.kv_shape(1) is None and cfg.state_shape(1) == [(3, 5, 6), (3, 5), (3,)]
    assert cfg.kv_shape(2) is None and cfg.state_shape(2) == [(4, 5, 3), (3, 12 + 2 * 2 * 5)]
    assert [cfg.source(i) for i in range(4)] == [0, 1, 2, 1] and cfg.state_shape(3) == cfg.state_shape(1)
    assert Z.ZuderaxConfig.from_dict({k: v for k, v in CFG.items() if k != "logit_scale"}).logit_scale == 1.0
    assert model_registry.architecture_of(CFG).name == "Zuderax" and "Zuderax" in model_registry.known_architectures()


@pytest.mark.parametrize("change,error", [
    (dict(SPACE, type="attention"), NotImplementedError),
    (dict(LATENT, mlp={"kind": "sparse", "ff": 3}), NotImplementedError),
    (dict(SPACE, mixer=dict(SPACE["mixer"], groups=3)), ValueError),
    (dict(SPACE, mixer=dict(SPACE["mixer"], norm_groups=5)), ValueError),
    (dict(LATENT, mixer=dict(LATENT["mixer"], rot={"base": 10.0, "dims": 6})), ValueError),
    (dict(MEMORY, mlp=dict(MEMORY["mlp"], router=dict(MEMORY["mlp"]["router"], groups={"count": 4, "keep": 2}))), ValueError),
    (dict(LATENT, weights_of=0), ValueError),                                     # itself
    (dict(LATENT, weights_of=9), ValueError),
    (dict(LATENT, weights_of=1), ValueError),                                     # another kind
])
def test_config_refuses_what_the_design_does_not_have(change, error):
    with pytest.raises(error):
        Z.ZuderaxConfig.from_dict(dict(CFG, layers=[change] + CFG["layers"][1:]))


def test_random_checkpoint_has_the_checkpoint_names():
    t = Z.random_checkpoint(Z.ZuderaxConfig.from_dict(CFG), seed=1)
    shapes = {k: tuple(v.shape) for k, v in t.items()}
    assert shapes["l0.norm1.alpha"] == () and shapes["l0.norm1.b"] == (24,) and "l2.norm2" not in t and shapes["final.norm.alpha"] == ()
    assert shapes["l0.mix.q"] == (20, 24) and shapes["l0.mix.dkv"] == (18, 24) and shapes["l0.mix.uk"] == (12, 14)
    assert shapes["l1.mix.q"] == (15, 24) and shapes["l1.mix.g"] == (18, 24) and shapes["l1.mix.i"] == (3, 24) and shapes["l1.mix.f.b"] == (3,)
    assert shapes["l1.mix.norm"] == (18,) and shapes["l2.mix.in"] == (12 + 12 + 20 + 4, 24) and shapes["l2.mix.conv"] == (32, 4)
    assert shapes["l1.mlp.router"] == (6, 24) and shapes["l1.mlp.correction"] == (6,) and shapes["l1.mlp.shared.sg"] == (1, 24)
    assert "l1.mlp.e5.down" in t and "l1.mlp.e6.up" not in t and not any(k.startswith("l3.") for k in t)
    logits = R.forward(CFG, t, [1, 5, 7, 2, 2, 18, 0, 3, 9, 11])
    assert logits.shape == (10, 19) and torch.isfinite(logits).all()


def test_oracle_rotation_and_masks():
    g = torch.Generator().manual_seed(0)
    x = torch.randn(5, 2, 8, generator=g, dtype=F64)
    turned = R.rotate_half(x, torch.arange(5), 4, 50.0)
    assert (turned[..., 4:] == x[..., 4:]).all() and (turned[0] == x[0]).all() and torch.allclose(turned.norm(dim=-1), x.norm(dim=-1))
    # one pair is (i, i + half): entry 1 of position 3 turns with entry 3 by 3 * 50^(-1/2)
    a = 3.0 * 50.0 ** -0.5
    assert torch.allclose(turned[3, 0, 1], x[3, 0, 1] * math.cos(a) - x[3, 0, 3] * math.sin(a))
    assert R.visible(9, 3)[5].tolist() == [False] * 3 + [True] * 3 + [False] * 3
    assert torch.equal(R.visible(7, 7), R.visible(7, 0))


def test_oracle_recurrences():
    g = torch.Generator().manual_seed(1)
    T, H, dk, dv = 12, 2, 3, 4
    q, k, v = (torch.randn(T, H, d, generator=g, dtype=F64) for d in (dk, dk, dv))
    i, f = R.capped_gates(3 * torch.randn(T, H, generator=g, dtype=F64), 3 * torch.randn(T, H, generator=g, dtype=F64), 2.0)
    assert i.abs().max() <= 2.0 and f.max() < 0
    # cut anywhere, the carried state continues the sequence
    o, end = R.matrix_memory(q, k, v, i, f)
    o1, s = R.matrix_memory(q[:5], k[:5], v[:5], i[:5], f[:5])
    o2, end2 = R.matrix_memory(q[5:], k[5:], v[5:], i[5:], f[5:], s)
    assert torch.allclose(torch.cat([o1, o2]), o) and all(torch.allclose(a, b) for a, b in zip(end, end2))
    # unrolled: weights exp(sum of f after s + i_s) over max(|.|, 1), whatever the running maximum is (up to the floor)
    F = torch.cumsum(f, 0)
    t = T - 1
    w = torch.exp(F[t] - F + i)                                            # [T, H]
    qk = torch.einsum("hd,shd->sh", q[t], k)
    num, den = torch.einsum("sh,shv->hv", w * qk, v), (w * qk).sum(0).abs().clamp(min=1.0)
    assert torch.allclose(o[t], num / den[:, None], rtol=1e-4)
    # state space: unrolled weights exp(-e^A sum of later steps) dt B.C, plus D x
    x, B, C = torch.randn(T, 4, dv, generator=g, dtype=F64), torch.randn(T, 2, 3, generator=g, dtype=F64), torch.randn(T, 2, 3, generator=g, dtype=F64)
    dt, A, D = torch.rand(T, 4, generator=g, dtype=F64), torch.randn(4, generator=g, dtype=F64), torch.randn(4, generator=g, dtype=F64)
    y, S = R.state_space(x, B, C, dt, A, D)
    c = torch.cumsum(dt, 0)
    for h in range(4):
        w = torch.exp(-torch.exp(A[h]) * (c[t, h] - c[:, h])) * dt[:, h] * (B[:, h // 2] @ C[t, h // 2])
        assert torch.allclose(y[t, h], w @ x[:, h] + D[h] * x[t, h])
    y1, s = R.state_space(x[:7], B[:7], C[:7], dt[:7], A, D)
    y2, S2 = R.state_space(x[7:], B[7:], C[7:], dt[7:], A, D, s)
    assert torch.allclose(torch.cat([y1, y2]), y) and torch.allclose(S, S2)
    w, b = torch.randn(6, 3, generator=g, dtype=F64), torch.randn(6, generator=g, dtype=F64)
    z = torch.randn(4, 6, generator=g, dtype=F64)
    conv = R.causal_conv(z, w, b)
    assert torch.allclose(conv[0], z[0] * w[:, 2] + b) and torch.allclose(conv[3], z[1] * w[:, 0] + z[2] * w[:, 1] + z[3] * w[:, 2] + b)


def test_oracle_routing():
    z = torch.logit(torch.tensor([[0.9, 0.1, 0.1, 0.6, 0.6, 0.1]], dtype=F64))
    ids, w = R.route(z, None, 2, 2, 1, 3.0)
    assert sorted(ids[0].tolist()) == [3, 4] and torch.allclose(w, torch.full((1, 2), 1.8, dtype=F64))
    # masked experts count as minus infinity: a negative choice score of a kept group beats them
    corr = torch.tensor([0.0, 0.0, 0.0, -5.0, -5.0, 9.0], dtype=F64)
    ids, w = R.route(z, corr, 3, 2, 1, 1.0)
    assert sorted(ids[0].tolist()) == [3, 4, 5] and torch.allclose(w.sort().values, torch.tensor([[0.1, 0.6, 0.6]], dtype=F64))
