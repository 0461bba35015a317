"""CPU: configuration, registry, pools and checkpoint layout of the Rufedra model class, and sanity of its oracle."""
import math

import pytest
import torch

import dgi_b200  # noqa: F401
from dgi_b200 import model_registry
from dgi_b200 import rufedra_layer as Q
from oracle import rufedra_ref as R

F64 = torch.float64
DELTA = {"type": "delta", "mixer": {"heads": 4, "kv_heads": 2, "dim": 5, "vdim": 6, "conv": 3}, "mlp": None}
LEFT = {"heads": 6, "kv_heads": 3, "dim": 8, "vdim": 8, "scale": 0.3, "mask": {"size": 7}, "rot": {"base": 100.0, "dims": 4}}
RIGHT = {"inner": 14, "state": 3, "dt_rank": 2, "conv": 4}
BOTH = {"type": "parallel", "mixer": {"left": LEFT, "right": RIGHT, "left_scale": 0.4, "right_scale": 1.1},
        "mlp": {"kind": "dense", "ff": 20}}
CFG = {"architecture": "Rufedra", "width": 24, "vocab": 19, "norm": {"eps": 1e-5}, "embedding": {"scale": 2.5}, "logit_scale": 0.7,
       "layers": [DELTA, BOTH, dict(DELTA, mlp={"kind": "dense", "ff": 9})]}


def test_config_names_pools_and_states():
    cfg = Q.RufedraConfig.from_dict(CFG)
    assert cfg.num_hidden_layers == 3 and cfg.hidden_size == 24 and cfg.vocab_size == 19
    assert cfg.logit_scale == 0.7 and cfg.embed_scale == 2.5 and cfg.num_attention_heads == 6
    assert cfg.kv_shape(0) is None and cfg.state_shape(0) == [(4, 5, 6), (2, 2 * 10 + 24)]
    assert cfg.kv_shape(1) == (3, 8, 8) and cfg.state_shape(1) == [(14, 3), (3, 14)]          # pages AND a state slot
    assert model_registry.architecture_of(CFG).name == "Rufedra" and "Rufedra" in model_registry.known_architectures()


@pytest.mark.parametrize("change,error", [
    (dict(DELTA, type="attention"), NotImplementedError),
    (dict(BOTH, mlp={"kind": "moe", "ff": 3}), NotImplementedError),
    (dict(DELTA, mixer=dict(DELTA["mixer"], kv_heads=3)), ValueError),
    (dict(BOTH, mixer=dict(BOTH["mixer"], left=dict(LEFT, kv_heads=4))), ValueError),
    (dict(BOTH, mixer=dict(BOTH["mixer"], left=dict(LEFT, vdim=6))), ValueError),             # the values ARE the keys
    (dict(BOTH, mixer=dict(BOTH["mixer"], left=dict(LEFT, rot={"base": 10.0, "dims": 10}))), ValueError),
    (dict(BOTH, mixer=dict(BOTH["mixer"], left=dict(LEFT, rot={"base": 10.0, "dims": 3}))), ValueError),
])
def test_config_refuses_what_the_design_does_not_have(change, error):
    with pytest.raises(error):
        Q.RufedraConfig.from_dict(dict(CFG, layers=[change] + CFG["layers"][1:]))


def test_random_checkpoint_has_the_checkpoint_names():
    t = Q.random_checkpoint(Q.RufedraConfig.from_dict(CFG), seed=1)
    shapes = {k: tuple(v.shape) for k, v in t.items()}
    assert shapes["l0.norm1b"] == (24,) and shapes["l0.ls1"] == (24,) and "l0.norm2" not in t and shapes["l2.ls2"] == (24,)
    assert shapes["l0.mix.q"] == (10, 24) and shapes["l0.mix.k.conv"] == (10, 3) and shapes["l0.mix.v.conv"] == (24, 3)
    assert shapes["l0.mix.a"] == (4, 24) and shapes["l0.mix.b"] == (4, 24) and shapes["l0.mix.norm"] == (6,)
    assert shapes["l0.mix.g"] == (24, 24) and shapes["l0.mix.o"] == (24, 24) and shapes["l0.mix.A_log"] == (4,)
    assert shapes["l1.mix.left.q"] == (48, 24) and shapes["l1.mix.left.k.b"] == (24,) and "l1.mix.left.v" not in t
    assert shapes["l1.mix.left.g"] == (48, 24) and shapes["l1.mix.left.o"] == (24, 48)
    assert shapes["l1.mix.right.in"] == (28, 24) and shapes["l1.mix.right.x"] == (8, 14) and shapes["l1.mix.right.dt"] == (14, 2)
    assert shapes["l1.mix.right.A_log"] == (14, 3) and shapes["l1.mix.right.conv.b"] == (14,) and shapes["l1.mlp.down"] == (24, 20)
    logits = R.forward(CFG, t, [1, 5, 7, 2, 2, 18, 0, 3, 9, 11])
    assert logits.shape == (10, 19) and torch.isfinite(logits).all()


def test_oracle_delta_rule():
    g = torch.Generator().manual_seed(1)
    T, H, dk, dv = 12, 2, 3, 4
    q, k = R.unit(torch.randn(T, H, dk, generator=g, dtype=F64)), R.unit(torch.randn(T, H, dk, generator=g, dtype=F64))
    v, dec, beta = torch.randn(T, H, dv, generator=g, dtype=F64), torch.rand(T, H, generator=g, dtype=F64), torch.rand(T, H, generator=g, dtype=F64)
    o, end = R.delta_rule(q, k, v, dec, beta)
    o1, s = R.delta_rule(q[:5], k[:5], v[:5], dec[:5], beta[:5])            # cut anywhere, the carried state continues
    o2, end2 = R.delta_rule(q[5:], k[5:], v[5:], dec[5:], beta[5:], s)
    assert torch.allclose(torch.cat([o1, o2]), o) and torch.allclose(end, end2)
    # the same as a product of matrices: S_t = (1 - beta k k^T) g S + beta k v^T
    for h in range(H):
        S = torch.zeros(dk, dv, dtype=F64)
        for t in range(T):
            kk = torch.outer(k[t, h], k[t, h])
            S = (torch.eye(dk, dtype=F64) - beta[t, h] * kk) @ (dec[t, h] * S) + beta[t, h] * torch.outer(k[t, h], v[t, h])
            assert torch.allclose(o[t, h], S.T @ q[t, h])
    # a full write without decay is read back exactly by its own key
    one = torch.ones(T, H, dtype=F64)
    o, _ = R.delta_rule(k, k, v, one, one)
    assert torch.allclose(o, v, atol=1e-3)


def test_oracle_selective_scan_and_attention():
    g = torch.Generator().manual_seed(2)
    T, I, N = 11, 3, 4
    x, dt = torch.randn(T, I, generator=g, dtype=F64), torch.rand(T, I, generator=g, dtype=F64)
    B, C = torch.randn(T, N, generator=g, dtype=F64), torch.randn(T, N, generator=g, dtype=F64)
    A, D = -torch.rand(I, N, generator=g, dtype=F64), torch.randn(I, generator=g, dtype=F64)
    y, S = R.selective_scan(x, dt, A, B, C, D)
    c, t = torch.cumsum(dt, 0), T - 1
    for i in range(I):                                                     # unrolled: exp(A sum of later steps) dt x B.C, plus D x
        w = torch.exp((c[t, i] - c[:, i])[:, None] * A[i]) * (dt[:, i] * x[:, i])[:, None] * B
        assert torch.allclose(y[t, i], (w @ C[t]).sum() + D[i] * x[t, i])
    y1, s = R.selective_scan(x[:4], dt[:4], A, B[:4], C[:4], D)
    y2, S2 = R.selective_scan(x[4:], dt[4:], A, B[4:], C[4:], D, s)
    assert torch.allclose(torch.cat([y1, y2]), y) and torch.allclose(S, S2)
    # rotation: entry 1 of position 3 turns with entry 3 by 3 * 50^(-1/2); a norm without a weight is the same before and after
    x = torch.randn(5, 2, 8, generator=g, dtype=F64)
    turned = R.rotate_half(x, torch.arange(5), 4, 50.0)
    a = 3.0 * 50.0 ** -0.5
    assert torch.allclose(turned[3, 0, 1], x[3, 0, 1] * math.cos(a) - x[3, 0, 3] * math.sin(a)) and (turned[..., 4:] == x[..., 4:]).all()
    assert torch.allclose(R.rms(turned, 0.1), R.rotate_half(R.rms(x, 0.1), torch.arange(5), 4, 50.0))
    assert R.visible(9, 3)[5].tolist() == [False] * 3 + [True] * 3 + [False] * 3
    # a window of one: every token attends to itself alone and reads its own projected key
    m = {"heads": 2, "kv_heads": 1, "dim": 4, "rot": {"base": 10.0, "dims": 4}, "scale": 1.0, "mask": {"size": 1}}
    W = 6
    t = {n: torch.randn(*s, generator=g, dtype=F64) for n, s in (("q", (8, W)), ("q.b", (8,)), ("k", (4, W)), ("k.b", (4,)), ("g", (8, W)), ("o", (W, 8)))}
    h = torch.randn(5, W, generator=g, dtype=F64)
    key = h @ t["k"].T + t["k.b"]
    want = (torch.cat([key, key], dim=1) * torch.sigmoid(h @ t["g"].T)) @ t["o"].T
    assert torch.allclose(R.key_value_attention(h, m, t, 1e-6), want)
    z, w = torch.randn(4, 6, generator=g, dtype=F64), torch.randn(6, 3, generator=g, dtype=F64)
    assert torch.allclose(R.causal_conv(z, w)[3], z[1] * w[:, 0] + z[2] * w[:, 1] + z[3] * w[:, 2])
    u = torch.linspace(-3, 3, 7, dtype=F64)
    assert torch.allclose(R.gelu_tanh(u), torch.nn.functional.gelu(u, approximate="tanh"))
