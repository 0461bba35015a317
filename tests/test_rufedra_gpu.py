"""GPU: the Rufedra model class on the ragged step engine against the plain float64 statement in oracle/rufedra_ref.py.

Small configurations with random weights; sizes are chosen so that nothing is a multiple of a warp, a page, a key tile or a scan
chunk by accident (one head, key sizes 1 / 6 / 33 / 40, value sizes 3 / 10 / 72, 1 / 2 / 3 / 5 taps, 1 / 3 / 5 / 19 states per
channel, step-size ranks 1 / 3, windows of 1, 9, 19 and longer than the sequence, rotations over none, a part and all of a head,
branch weights that are negative or zero, layers without a feed-forward).  Where random weights would hide a fault the inputs are
made so that it shows: one key dominates just inside and just outside a window, keys of the delta rule point almost the same way,
decays are close to 1 and close to 0, one far key among hundreds is the only one a query matches.
"""
import math

import pytest
import torch

import dgi_b200  # noqa: F401
from oracle import rufedra_ref as R

pytestmark = pytest.mark.gpu

DEV = "cuda:0"
F64 = torch.float64


def delta(heads, kv_heads, dim, vdim, conv, ff=None):
    return {"type": "delta", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "conv": conv},
            "mlp": {"kind": "dense", "ff": ff} if ff else None}


def parallel(left, right, scales=(0.7, 0.8), ff=None):
    H, G, dim, size, base, dims, scale = left
    inner, state, rank, conv = right
    return {"type": "parallel", "mlp": {"kind": "dense", "ff": ff} if ff else None,
            "mixer": {"left": {"heads": H, "kv_heads": G, "dim": dim, "vdim": dim, "mask": {"size": size}, "scale": scale,
                               "rot": {"base": base, "dims": dims}},
                      "right": {"inner": inner, "state": state, "dt_rank": rank, "conv": conv},
                      "left_scale": scales[0], "right_scale": scales[1]}}


def model(width, vocab, layers, eps=1e-5, emb=1.0, logit=1.0):
    return {"architecture": "Rufedra", "width": width, "vocab": vocab, "norm": {"eps": eps}, "embedding": {"scale": emb},
            "logit_scale": logit, "layers": layers}


CFG_A = model(50, 53, [      # sizes off every grid
    parallel((6, 2, 10, 9, 50.0, 6, 0.4), (30, 5, 3, 5), ff=27),
    delta(6, 3, 6, 10, 5),
    delta(3, 1, 33, 3, 2, ff=11),
    parallel((3, 3, 7, 19, 900.0, 0, 0.3), (13, 19, 1, 1), scales=(-0.5, 1.3)),
    parallel((4, 1, 12, 300, 20.0, 12, 0.25), (21, 1, 2, 3), scales=(1.0, 0.0), ff=9),
    parallel((2, 1, 4, 3, 20.0, 2, 0.5), (9, 3, 2, 2), scales=(0.0, 0.6)),
], emb=3.0, logit=0.3)
CFG_B = model(64, 41, [      # sizes the tensor-core kernels take in 16-bit storage
    delta(4, 2, 32, 48, 3),
    parallel((12, 3, 32, 40, 200.0, 16, 0.2), (96, 16, 8, 4), ff=96),
    delta(2, 2, 128, 64, 4, ff=40),
    parallel((20, 1, 16, 19, 200.0, 16, 0.3), (40, 24, 4, 2), scales=(0.9, -0.4)),
    delta(2, 1, 160, 24, 1),
], eps=1e-6, logit=0.7)
CFG_C = model(8, 11, [parallel((1, 1, 2, 1, 10.0, 2, 1.0), (1, 1, 1, 1)), delta(1, 1, 1, 1, 1, ff=3)], eps=1e-6)   # the smallest
CFG_D = model(48, 37, [delta(4, 4, 16, 32, 4, ff=64), delta(2, 1, 72, 72, 3)], eps=1e-6)                     # no pages at all


def build(cfg_raw, dtype=torch.float32, seed=0, max_tokens=512, max_seqs=4, tensors=None):
    from dgi_b200 import rufedra_layer as Q
    from dgi_b200.ragged_engine import RaggedStepEngine

    cfg = Q.RufedraConfig.from_dict(cfg_raw)
    tensors = tensors or Q.random_checkpoint(cfg, seed=seed)
    shards = Q.build_shards(cfg, tensors, [(0, cfg.num_hidden_layers)], DEV, dtype)
    return RaggedStepEngine(shards, max_tokens=max_tokens, max_seqs=max_seqs), tensors


def tokens(n, vocab, seed):
    return torch.randint(0, vocab, (n,), generator=torch.Generator().manual_seed(seed)).tolist()


def whole(engine, rid, toks, want=None):
    want = list(range(len(toks))) if want is None else want
    out = engine.step([(rid, toks, want)]).cpu()
    engine.finish(rid)
    return out


def close(got, ref, tol):
    err = (got.to(F64) - ref.to(F64)).abs().max().item()
    assert err <= tol * max(1.0, ref.abs().max().item()), f"max abs error {err}"


def rounding_close(got, ref, cfg=None, median=0.04, tail=0.15):
    """16-bit storage against a wider statement, row by row (error rms over the statement's rms).  Read-outs of one or three values
    that are made unit-RMS (CFG_A, CFG_C) turn by large angles under rounding where they are near zero: a few such rows may
    differ more (the statement with its products rounded to 16 bits does the same)."""
    row = (got.to(F64) - ref.to(F64)).pow(2).mean(dim=1).sqrt() / ref.to(F64).pow(2).mean().sqrt()
    assert row.median() <= median, f"median row error {row.median().item()}"
    allowed = 0.06 * row.numel() if cfg is CFG_A or cfg is CFG_C else 0
    assert (row > tail).sum() <= allowed, f"{(row > tail).sum().item()} of {row.numel()} rows over {tail}, worst {row.max().item()}"


def seqs_of(spans):
    return torch.tensor(spans, dtype=torch.int32, device=DEV)


DT = pytest.mark.parametrize("dt,tol", [(torch.float32, 3e-6), (torch.bfloat16, 1e-2)], ids=["fp32", "bf16"])


# ---- row-wise pieces ---------------------------------------------------------------------------------------------------
@DT
@pytest.mark.parametrize("n,W", [(5, 56), (3, 7), (2, 1032), (2, 2048), (3, 4096), (1, 8192), (2, 9000)])
def test_residual_update_normed_on_both_sides(dt, tol, n, W):
    from dgi_b200 import mixer_ops as M

    g = torch.Generator().manual_seed(W)
    x = 4.0 * torch.randn(n, W, generator=g)
    y = (3.0 * torch.randn(n, W + 8, generator=g)).to(dt)[:, :W]
    w, ls, wn = (torch.randn(W, generator=g).to(dt) for _ in range(3))
    for branch, scale, sign, nxt in ((y, ls, 1.0, wn), (y.float(), None, -1.0, wn), (y, ls, 1.0, None)):
        xd = x.to(DEV).clone()
        out = M.sandwich_residual(xd, branch.to(DEV), w.to(DEV), None if scale is None else scale.to(DEV), 0.03,
                                  None if nxt is None else nxt.to(DEV), 0.2, sign=sign)
        want = x.to(F64) + sign * R.rms(branch.to(F64), 0.03) * w.to(F64) * (1.0 if scale is None else scale.to(F64))
        close(xd.cpu(), want, 2e-6)                                     # the residual stays fp32
        if nxt is None:
            assert out is None
        else:
            assert out.dtype == dt
            close(out.cpu(), R.rms(want, 0.2) * wn.to(F64), tol)


@DT
@pytest.mark.parametrize("ff", [5, 16, 40])
def test_gelu_glu(dt, tol, ff):
    from dgi_b200 import mixer_ops as M

    gu = 3.0 * torch.randn(9, 2 * ff, generator=torch.Generator().manual_seed(ff))
    gu[0, :2], gu[1, :2] = torch.tensor([30.0, -30.0]), torch.tensor([0.0, 1e-3])       # far out and near zero
    gu = gu.to(dt)
    close(M.gelu_glu(gu.to(DEV)).cpu(), R.gelu_tanh(gu[:, :ff].to(F64)) * gu[:, ff:].to(F64), tol)


@DT
@pytest.mark.parametrize("H,G,dk,dims", [(6, 2, 10, 6), (3, 3, 7, 0), (4, 1, 64, 64), (1, 1, 2, 2), (9, 3, 40, 16)])
def test_rotated_unit_keys_beside_the_projected_keys_as_values(dt, tol, H, G, dk, dims):
    from dgi_b200 import mixer_ops as M
    from dgi_b200.fibirax_layer import wavelength_scaled_frequencies

    g = torch.Generator().manual_seed(H + dk)
    n, bs, nb = 21, 16, 3
    proj = torch.randn(n, (H + G) * dk, generator=g).to(dt)
    pos = torch.randint(0, 5000, (n,), generator=g).to(torch.int32)
    slots = torch.randperm(nb * bs, generator=g)[:n].to(torch.int64)
    kp, vp = (torch.zeros((nb, G, bs, dk), dtype=dt, device=DEV) for _ in range(2))
    dev = proj.to(DEV)
    freqs = wavelength_scaled_frequencies(dims, 300.0, None)
    q, k = dev[:, :H * dk], dev[:, H * dk:]
    M.qknorm_rotary_append(q, k, k, None, None, 0.05, freqs.to(DEV) if dims else None, kp, vp, slots.to(DEV), pos.to(DEV), H,
                           interleaved=False, unit_norm=True)
    want = R.rms(R.rotate_half(proj.to(F64).reshape(n, H + G, dk), pos, dims, 300.0), 0.05)
    close(q.cpu().reshape(n, H, dk), want[:, :H], tol)
    rows = lambda pool: pool.permute(0, 2, 1, 3).reshape(nb * bs, G, dk)[slots.to(DEV)].cpu()       # noqa: E731
    close(rows(kp), want[:, H:], tol)
    assert torch.equal(rows(vp).reshape(n, G * dk), proj[:, H * dk:])       # values: the projection itself


# ---- attention with a gate per output channel, heads on the rows ---------------------------------------------------------
def _pages(k, v, bs, seed):
    """``k``, ``v`` ``[T, G, d]`` in shuffled pages: ``(k pool, v pool, block table)``."""
    T, G = k.shape[:2]
    nb = (T + bs - 1) // bs
    table = torch.randperm(nb + 2, generator=torch.Generator().manual_seed(seed))[:nb]
    pools = []
    for x in (k, v):
        pool = torch.zeros(nb + 2, G, bs, x.shape[2], dtype=x.dtype)
        for t in range(T):
            pool[table[t // bs], :, t % bs] = x[t]
        pools.append(pool)
    return pools[0], pools[1], table.to(torch.int32)


LAYOUTS = [(6, 2, 16, 16), (40, 2, 32, 24), (40, 1, 32, 24), (8, 8, 16, 8), (12, 4, 64, 64), (20, 1, 16, 64), (16, 2, 128, 128), (3, 1, 16, 8)]


@pytest.mark.parametrize("H,G,dk,dv", LAYOUTS)
@pytest.mark.parametrize("path", ["rows-fp32", "prompt-bf16", "prompt-fp16", "single-bf16", "single-heads-bf16", "single-heads-fp16"])
@pytest.mark.parametrize("window", [0, 37])
def test_attention_with_a_gate_per_channel_or_head(H, G, dk, dv, path, window):
    from dgi_b200 import mixer_ops as M

    kind, name = path.rsplit("-", 1)
    if kind == "single-heads" and G > 1:
        pytest.skip("heads go on the rows over one kv head")
    dt = {"fp32": torch.float32, "bf16": torch.bfloat16, "fp16": torch.float16}[name]
    g = torch.Generator().manual_seed(H * dk + dv)
    T, bs, scale = 333, 16, 1.0 / math.sqrt(dk)
    k, v = torch.randn(T, G, dk, generator=g).to(dt), torch.randn(T, G, dv, generator=g).to(dt)
    single = kind.startswith("single")
    pos = torch.tensor([0, 15, 16, 31, 36, 37, 38, 200, 332]) if single else torch.arange(290, 333)
    n = len(pos)
    q = torch.randn(n, H, dk, generator=g).to(dt)
    k[5] = 2.5 * q[0, 0]                                           # keys that stand out
    k[300] = 2.5 * q[-1, 0]
    gates = {"channel": torch.randn(n, H * dv, generator=g).to(dt), "head": torch.randn(n, H, generator=g).to(dt), "none": None}
    sink = torch.randn(H, generator=g)
    of = torch.arange(H) // (H // G)
    s = torch.einsum("ihd,jhd->hij", q.to(F64), k.to(F64)[:, of]) * scale
    d = pos[:, None] - torch.arange(T)[None]
    s = s.masked_fill(~((d >= 0) & ((d < window) if window else (d >= 0)))[None], float("-inf"))
    kp, vp, table = _pages(k, v, bs, 3)
    kp, vp = kp.to(DEV), vp.to(DEV)
    for gk, gate in gates.items():
        for with_sink in (False, True):
            extra = sink.to(F64)[:, None, None].expand(H, n, 1) if with_sink else torch.full((H, n, 1), float("-inf"), dtype=F64)
            p = torch.softmax(torch.cat([s, extra], dim=-1), dim=-1)[..., :T]
            want = torch.einsum("hij,jhd->ihd", p, v.to(F64)[:, of])
            if gk == "channel":
                want = want * torch.sigmoid(gate.to(F64)).reshape(n, H, dv)
            elif gk == "head":
                want = want * torch.sigmoid(gate.to(F64))[:, :, None]
            rows = n if single else 1
            tables = table[None].expand(rows, -1).contiguous().to(DEV)
            out = torch.full((n, H * dv + 8), 7.0, dtype=dt, device=DEV)
            view = out[:, :H * dv].unflatten(1, (H, dv))
            kw = dict(window=window, gate=None if gate is None else gate.to(DEV), sink=sink.to(DEV) if with_sink else None)
            tp = pos.to(torch.int32).to(DEV)
            if kind == "rows":
                M.mixed_paged_attention(view, q.to(DEV), kp, vp, tables, torch.zeros(n, dtype=torch.int32, device=DEV), tp, scale, **kw)
            else:
                if single:
                    tiles = [(i, 1, i) for i in range(n)]
                else:
                    tiles = [(i, min(16, n - i), 0) for i in range(0, n, 16)]
                if kind == "single-heads":
                    assert M.heads_as_rows_supported(H, dk, dv, dt)
                for ctx in (0, 333):                                  # one CTA per tile, and the keys divided over several
                    M.mixed_prompt_attention(view, q.to(DEV), kp, vp, tables, torch.tensor(tiles, dtype=torch.int32, device=DEV),
                                             tp, scale, max_context=ctx, heads_as_rows=kind == "single-heads", **kw)
                    close(out[:, :H * dv].cpu().reshape(n, H, dv), want, 1.5e-2)
            close(out[:, :H * dv].cpu().reshape(n, H, dv), want, 1e-5 if dt == torch.float32 else 1.5e-2)
            assert (out[:, H * dv:] == 7.0).all()


# ---- the delta rule --------------------------------------------------------------------------------------------------------
def _delta_case(H, G, dk, dv, n, dt, seed, kind):
    g = torch.Generator().manual_seed(seed)
    x = torch.randn(n, 2 * G * dk + H * dv + 8, generator=g)
    z = torch.randn(n, 2 * H, generator=g)
    if kind == "alike":                       # keys point almost the same way and every write is nearly complete
        x[:, G * dk:2 * G * dk] = 2.0 + 0.1 * x[:, G * dk:2 * G * dk]
        z[:, :H] += 4.0
    z[:, H:] += {"slow": -5.0, "alike": -5.0, "mixed": 0.0}[kind]
    dt_bias, a_log = torch.randn(H, generator=g), torch.randn(H, generator=g)
    z[n // 3, H:] = 60.0                      # everything before this token is forgotten
    return x.to(dt), z.to(dt), dt_bias.to(dt), a_log.to(dt)


def _delta_reference(x, z, dt_bias, a_log, H, G, dk, dv):
    n = x.shape[0]
    of = torch.arange(H) // (H // G)
    q = R.unit(x[:, :G * dk].to(F64).reshape(n, G, dk))[:, of] * 0.6
    k = R.unit(x[:, G * dk:2 * G * dk].to(F64).reshape(n, G, dk))[:, of]
    v = x[:, 2 * G * dk:2 * G * dk + H * dv].to(F64).reshape(n, H, dv)
    decay = torch.exp(-torch.exp(a_log.to(F64)) * R.softplus(z[:, H:].to(F64) + dt_bias.to(F64)))
    return R.delta_rule(q, k, v, decay, torch.sigmoid(z[:, :H].to(F64)))


def _delta_run(M, x, z, dt_bias, a_log, state, seqs, H, G, dk, dv, max_count):
    return M.delta_scan(x[:, :G * dk], x[:, G * dk:2 * G * dk], x[:, 2 * G * dk:2 * G * dk + H * dv], z[:, :H], z[:, H:], dt_bias,
                        a_log, state, seqs, G, R.UNIT_EPS, 0.6, max_count=max_count)


DELTAS = [(6, 3, 6, 10), (3, 1, 33, 3), (4, 2, 32, 48), (2, 2, 128, 64), (2, 1, 160, 24), (1, 1, 1, 1), (4, 4, 64, 128), (2, 1, 256, 100),
          (8, 2, 128, 32), (2, 2, 72, 40),
          (76, 2, 20, 40), (80, 1, 128, 72), (75, 75, 130, 64)]      # enough heads for the widest blocks of value columns


@pytest.mark.parametrize("H,G,dk,dv", DELTAS)
@pytest.mark.parametrize("kind", ["mixed", "slow", "alike"])
@pytest.mark.parametrize("path", ["tokens-fp32", "tokens-bf16", "tokens-fp16", "chunks-bf16"])
def test_delta_rule_with_one_decay_per_head_over_portions_beside_another_sequence(H, G, dk, dv, kind, path):
    from dgi_b200 import mixer_ops as M

    chunks = path.startswith("chunks")
    dt = {"fp32": torch.float32, "bf16": torch.bfloat16, "fp16": torch.float16}[path.split("-")[1]]
    n = 330
    x, z, dt_bias, a_log = _delta_case(H, G, dk, dv, n, dt, H * dk + dv, kind)
    want, want_S = _delta_reference(x, z, dt_bias, a_log, H, G, dk, dv)
    state = torch.full((3, H, dk, dv), float("nan"), device=DEV)       # a fresh sequence never reads its slot
    dx, dz, db, da = (t.to(DEV) for t in (x, z, dt_bias, a_log))
    at, got = 0, []
    # 16-bit inputs are exact here; everything between them and the read-outs is 32-bit, or its equivalent in split products
    tol = 2e-5 if not chunks else 6e-5
    for cut in (150, 1, 2, 63, 64, 7, 43):
        cat = lambda t: torch.cat([t[:5], t[at:at + cut]])             # noqa: E731  a second, fresh sequence in front
        o = _delta_run(M, cat(dx), cat(dz), db, da, state, seqs_of([(0, 5, 0, 1), (5, cut, 2, int(at == 0))]), H, G, dk, dv,
                       max(cut, 16) if chunks else 0)
        close(o[:5].cpu(), want[:5], tol)
        got.append(o[5:])
        at += cut
    close(torch.cat(got).cpu(), want, tol)
    close(state[2].cpu(), want_S, tol)
    assert torch.isnan(state[1]).all()


@pytest.mark.parametrize("H,G,dk,dv", DELTAS)
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
def test_single_token_delta_steps_equal_the_scan(H, G, dk, dv, dt):
    """Sequences in shuffled slots, one of them fresh."""
    from dgi_b200 import mixer_ops as M

    n = 5
    x, z, dt_bias, a_log = (t.to(DEV) for t in _delta_case(H, G, dk, dv, n, dt, 7, "mixed"))
    spans = seqs_of([(0, 1, 3, 0), (1, 1, 0, 1), (2, 1, 5, 0), (3, 1, 1, 0), (4, 1, 2, 0)])
    a = torch.randn(6, H, dk, dv, generator=torch.Generator().manual_seed(dk)).to(DEV)
    b = a.clone()
    o = _delta_run(M, x, z, dt_bias, a_log, a, spans, H, G, dk, dv, 0)
    o2 = _delta_run(M, x, z, dt_bias, a_log, b, spans, H, G, dk, dv, 1)
    close(o2.cpu(), o.cpu(), 2e-5)
    close(b.cpu(), a.cpu(), 2e-5)
    assert torch.equal(a[4], b[4])


def test_a_decay_per_channel_that_is_the_same_in_all_channels_equals_a_decay_per_head():
    from dgi_b200 import mixer_ops as M

    H, G, dk, dv, n = 4, 2, 12, 20, 40
    x, z, dt_bias, a_log = (t.to(DEV) for t in _delta_case(H, G, dk, dv, n, torch.float32, 1, "mixed"))
    spans = seqs_of([(0, n, 0, 1)])
    s1, s2 = torch.zeros(1, H, dk, dv, device=DEV), torch.zeros(1, H, dk, dv, device=DEV)
    o1 = _delta_run(M, x, z, dt_bias, a_log, s1, spans, H, G, dk, dv, 0)
    o2 = M.delta_scan(x[:, :G * dk], x[:, G * dk:2 * G * dk], x[:, 2 * G * dk:2 * G * dk + H * dv], z[:, :H],
                      z[:, H:].repeat_interleave(dk, dim=1), dt_bias.repeat_interleave(dk), a_log, s2, spans, G, R.UNIT_EPS, 0.6)
    assert torch.equal(o1, o2) and torch.equal(s1, s2)


# ---- the selective scan ------------------------------------------------------------------------------------------------------
SELECTIVE = [(30, 5), (13, 19), (21, 1), (9, 3), (96, 16), (40, 24), (256, 64), (130, 100), (8, 256), (64, 8), (200, 12)]


@pytest.mark.parametrize("inner,N", SELECTIVE)
@pytest.mark.parametrize("dt,tol", [(torch.float32, 1e-5), (torch.bfloat16, 1e-2), (torch.float16, 2e-3)], ids=["fp32", "bf16", "fp16"])
@pytest.mark.parametrize("slow", [False, True])
def test_selective_scan_over_portions_slots_and_single_tokens(inner, N, dt, tol, slow):
    from dgi_b200 import mixer_ops as M

    g = torch.Generator().manual_seed(inner + N)
    n, pad = 200, 8
    wide = torch.randn(n, 3 * (inner + pad), generator=g).to(dt)
    x, dtl, z = (wide[:, i * (inner + pad):i * (inner + pad) + inner] for i in range(3))
    bc = torch.randn(n, 2 * N + 4, generator=g).to(dt)
    B, C = bc[:, :N], bc[:, N + 4:]
    bias = torch.randn(inner, generator=g) - (5.0 if slow else 1.0)
    a_log, D = torch.randn(inner, N, generator=g) - (2.0 if slow else 0.0), torch.randn(inner, generator=g)
    y, S = R.selective_scan(x.to(F64), R.softplus(dtl.to(F64) + bias.to(F64)), -torch.exp(a_log.to(F64)), B.to(F64), C.to(F64), D.to(F64))
    want = 0.7 * y * R.silu(z.to(F64))
    state = torch.full((3, inner, N), float("nan"), device=DEV)
    dw, dbc = wide.to(DEV), bc.to(DEV)
    consts = [t.to(DEV) for t in (bias, -torch.exp(a_log), D)]
    out = torch.full((n + 3, inner + 6), 9.0, dtype=dt, device=DEV)
    at = 0
    for cut in (70, 1, 1, 2, 33, 32, 31, 30):
        first = 3 if cut == 33 else 0                                     # sometimes a second, fresh sequence in front
        rows = torch.cat([torch.arange(first), torch.arange(at, at + cut)]).to(DEV)
        w, b = dw[rows], dbc[rows]
        spans = [(first, cut, 2, int(at == 0))] if not first else [(0, 3, 0, 1), (3, cut, 2, 0)]
        sl = [w[:, i * (inner + pad):i * (inner + pad) + inner] for i in range(3)]
        o = out[at:at + cut + first, 2:2 + inner]
        M.selective_scan(sl[0], sl[1], b[:, :N], b[:, N + 4:], sl[2], *consts, state, seqs_of(spans), gain=0.7, out=o,
                         max_count=max(cut, first))
        if first:
            close(o[:3].cpu(), want[:3], tol)
            out[at:at + cut] = out[at + 3:at + 3 + cut].clone()
        at += cut
    close(out[:n, 2:2 + inner].cpu(), want, tol)
    assert (out[:n, :2] == 9.0).all() and (out[:n, 2 + inner:] == 9.0).all()
    close(state[2].cpu(), S, 1e-5 if dt == torch.float32 else 5e-5)
    assert torch.isnan(state[1]).all()


@pytest.mark.parametrize("inner,N", [(520, 16), (515, 3), (1030, 12), (300, 136)])
@pytest.mark.parametrize("dt,tol", [(torch.float32, 1e-5), (torch.bfloat16, 1e-2)], ids=["fp32", "bf16"])
def test_selective_steps_of_many_sequences(inner, N, dt, tol):
    """Slots in reverse, every third sequence fresh."""
    from dgi_b200 import mixer_ops as M

    g = torch.Generator().manual_seed(inner)
    n = 230
    x, dtl, z = (torch.randn(n, inner, generator=g).to(dt) for _ in range(3))
    B, C = torch.randn(n, N, generator=g).to(dt), torch.randn(n, N, generator=g).to(dt)
    bias, rates, D = torch.randn(inner, generator=g) - 1.0, -torch.rand(inner, N, generator=g), torch.randn(inner, generator=g)
    fresh = torch.arange(n) % 3 == 0
    state = torch.randn(n, inner, N, generator=g)
    S = state.flip(0).to(F64) * (~fresh)[:, None, None]
    step = R.softplus(dtl.to(F64) + bias.to(F64))
    S = torch.exp(step[:, :, None] * rates.to(F64)) * S + (step * x.to(F64))[:, :, None] * B.to(F64)[:, None, :]
    want = ((S * C.to(F64)[:, None, :]).sum(-1) + D.to(F64) * x.to(F64)) * R.silu(z.to(F64))
    dev = state.to(DEV)
    spans = seqs_of([(i, 1, n - 1 - i, int(fresh[i])) for i in range(n)])
    out = M.selective_scan(*(t.to(DEV) for t in (x, dtl, B, C, z, bias, rates, D)), dev, spans, max_count=1)
    close(out.cpu(), want, tol)
    close(dev.cpu().flip(0), S, 1e-5)


def test_selective_state_keeps_32_bit_accuracy_over_thousands_of_slow_tokens():
    from dgi_b200 import mixer_ops as M

    n, inner, N = 4000, 4, 8
    g = torch.Generator().manual_seed(0)
    x, dtl, z, B, C = (torch.randn(n, w, generator=g) for w in (inner, inner, inner, N, N))
    bias, a_log, D = torch.full((inner,), -5.0), torch.full((inner, N), -3.0), torch.zeros(inner)
    y, S = R.selective_scan(x.to(F64), R.softplus(dtl.to(F64) - 5.0), -torch.exp(a_log.to(F64)), B.to(F64), C.to(F64), D.to(F64))
    state = torch.zeros(1, inner, N, device=DEV)
    out = M.selective_scan(*(t.to(DEV) for t in (x, dtl, B, C, z, bias, -torch.exp(a_log), D)), state, seqs_of([(0, n, 0, 1)]), max_count=n)
    close(out.cpu(), y * R.silu(z.to(F64)), 4e-6)
    close(state[0].cpu(), S, 4e-6)


# ---- attention edges -----------------------------------------------------------------------------------------------------------
def _edge_model(window, heads=4, kv=2, dk=16):
    """A one-layer model with one number of interest per token: the query is a constant, a marked token's key points its way and
    all others away from it, in dimensions the rotation leaves alone, so a marked token takes all the weight wherever it is
    visible - and its value, being the key itself, says so."""
    W = 24
    cfg = model(W, 4, [parallel((heads, kv, dk, window, 100.0, 8, 1.5), (8, 2, 1, 2), scales=(1.0, 0.3))], eps=1e-6)
    g = torch.Generator().manual_seed(window)
    f = lambda *s: torch.randn(*s, generator=g) / math.sqrt(s[-1])        # noqa: E731
    t = {"embed": torch.zeros(4, W), "head": f(4, W), "final.norm": torch.ones(W)}
    t["embed"][:, 0] = 3.0                                                # every token: a constant channel
    t["embed"][1, 1], t["embed"][0, 2], t["embed"][2, 3], t["embed"][3, 4] = 3.0, 3.0, 3.0, 3.0
    for name in ("norm1", "norm1b", "ls1"):
        t["l0." + name] = torch.ones(W)
    q, k = torch.zeros(heads * dk, W), torch.zeros(kv * dk, W)
    for h in range(heads):
        q[h * dk + 8, 0] = 4.0
    for h in range(kv):
        k[h * dk + 8, 1], k[h * dk + 9, 2], k[h * dk + 10, 3], k[h * dk + 11, 4] = 2.0, 2.0, 2.0, 2.0
    p = "l0.mix.left."
    t.update({p + "q": q, p + "k": k, p + "q.b": torch.zeros(heads * dk), p + "k.b": 0.05 * torch.ones(kv * dk),
              p + "g": f(heads * dk, W), p + "o": f(W, heads * dk)})
    p = "l0.mix.right."
    t.update({p + "in": f(16, W), p + "conv": f(8, 2), p + "conv.b": torch.zeros(8), p + "x": f(5, 8), p + "dt": f(8, 1),
              p + "dt.b": torch.zeros(8), p + "A_log": torch.zeros(8, 2), p + "D": torch.ones(8), p + "o": f(W, 8)})
    return cfg, {k: v.to(torch.bfloat16) for k, v in t.items()}


@pytest.mark.parametrize("dt,tol", [(torch.float32, 2e-5), (torch.bfloat16, 0.05)], ids=["fp32", "bf16"])
@pytest.mark.parametrize("window", [1, 2, 15, 16, 17, 33, 64, 100])
def test_a_dominating_key_just_inside_and_just_outside_the_window_in_prompts_and_decoding(dt, tol, window):
    cfg, t = _edge_model(window)
    toks = [0, 2, 3] * 70
    for p in (3, 14, 15, 16, 31, 32, 47, 90):
        toks[p] = 1
    ref = R.forward(cfg, t, toks)
    for wrong in (window - 1, window + 1):       # a window off by one token would show
        if wrong >= 1:
            other = model(24, 4, [parallel((4, 2, 16, wrong, 100.0, 8, 1.5), (8, 2, 1, 2), scales=(1.0, 0.3))], eps=1e-6)
            assert (R.forward(other, t, toks) - ref).abs().max() > 0.2
    engine, _ = build(cfg, dtype=dt, tensors=t, max_tokens=256, max_seqs=2)
    close(whole(engine, "a", toks), ref, tol)
    got = [engine.step([("b", toks[:61], list(range(61)))])]
    for p in range(61, 200):
        got.append(engine.step([("b", [toks[p]], [0])]))
    engine.finish("b")
    close(torch.cat(got).cpu(), ref[:200], tol)


def test_one_far_key_among_hundreds_inside_a_long_window_bf16():
    cfg, t = _edge_model(700)
    toks = [0, 2, 3, 2, 0] * 160
    toks[37] = 1
    ref = R.forward(cfg, t, toks)
    assert (ref[736] - ref[737]).abs().max() > 0.2           # 737 no longer sees it
    engine, _ = build(cfg, dtype=torch.bfloat16, tensors=t, max_tokens=1024, max_seqs=1)
    want = [36, 37, 300, 735, 736, 737, 738, 799]
    close(whole(engine, "a", toks, want), ref[want], 0.05)


def test_what_the_delta_state_keeps_from_hundreds_of_tokens_ago():
    """Slow decay, one token written into an orthogonal direction and read back 500 tokens later, in prompts and decoding."""
    from dgi_b200 import mixer_ops as M

    H, G, dk, dv, n = 2, 1, 16, 8, 520
    g = torch.Generator().manual_seed(4)
    x = torch.randn(n, 2 * G * dk + H * dv, generator=g)
    x[:, dk + 15] = 0.0                                       # no other key touches direction 15
    x[3, dk:2 * dk] = 0.0
    x[3, dk + 15] = 5.0
    x[510, :dk] = 0.0
    x[510, 15] = 1.0                                          # asks for token 3 alone
    z = torch.zeros(n, 2 * H)
    z[:, H:] = -9.0
    x, z = x.to(torch.bfloat16), z.to(torch.bfloat16)
    const = torch.zeros(H, dtype=torch.bfloat16)
    want, _ = _delta_reference(x, z, const, const, H, G, dk, dv)
    assert want[510].abs().max() > 0.1
    state = torch.zeros(1, H, dk, dv, device=DEV)
    dx, dz, c = x.to(DEV), z.to(DEV), const.to(DEV)
    o = [_delta_run(M, dx[:500], dz[:500], c, c, state, seqs_of([(0, 500, 0, 1)]), H, G, dk, dv, 500)]
    for p in range(500, n):
        o.append(_delta_run(M, dx[p:p + 1], dz[p:p + 1], c, c, state, seqs_of([(0, 1, 0, 0)]), H, G, dk, dv, 1))
    close(torch.cat(o).cpu(), want, 6e-5)


# ---- the model through the engine ------------------------------------------------------------------------------------------
ALL = pytest.mark.parametrize("cfg", [CFG_A, CFG_B, CFG_C, CFG_D], ids=["A", "B", "C", "D"])
AB = pytest.mark.parametrize("cfg", [CFG_A, CFG_B], ids=["A", "B"])


@ALL
def test_whole_prompt_fp32(cfg):
    engine, tensors = build(cfg)
    toks = tokens(90, cfg["vocab"], 11)
    layers = []
    ref = R.forward(cfg, tensors, toks, trace=layers)
    engine.layer_trace = []
    got = whole(engine, "a", toks)
    for mine, theirs in zip(engine.layer_trace, layers):                    # the residual after every layer
        close(mine.cpu(), theirs, 5e-5)
    engine.layer_trace = None
    close(got, ref, 5e-5)
    one = tokens(1, cfg["vocab"], 12)                                       # the first token alone
    close(whole(engine, "b", one), R.forward(cfg, tensors, one), 5e-5)


@ALL
def test_whole_prompt_bf16(cfg):
    engine, tensors = build(cfg, dtype=torch.bfloat16)
    toks = tokens(70, cfg["vocab"], 13)
    rounding_close(whole(engine, "a", toks), R.forward(cfg, tensors, toks), cfg)


@ALL
def test_prefill_then_long_decode_matches_the_whole_prompt(cfg):
    engine, tensors = build(cfg)
    toks = tokens(120, cfg["vocab"], 14)
    ref = R.forward(cfg, tensors, toks)
    got = [engine.step([("a", toks[:30], list(range(30)))])]
    for t in range(30, len(toks)):                               # 90 decoded tokens: the windows pass over them
        got.append(engine.step([("a", [toks[t]], [0])]))
    engine.finish("a")
    close(torch.cat(got).cpu(), ref, 5e-5)
    got = [engine.step([("b", [t], [0])]) for t in toks[:40]]    # decoding from the very first token, in a used slot
    engine.finish("b")
    close(torch.cat(got).cpu(), ref[:40], 5e-5)


@AB
def test_portions_of_any_size_down_to_two_tokens(cfg):
    engine, tensors = build(cfg)
    toks = tokens(131, cfg["vocab"], 15)
    ref = R.forward(cfg, tensors, toks)
    for cuts in ([2, 2, 13, 3, 16, 17, 2, 31, 33, 2, 1, 9], [64, 2, 65], [15, 1, 16, 1, 31, 1, 2, 64], [8, 1, 9, 1, 10, 102]):
        got, at = [], 0
        for c in cuts:
            c = min(c, len(toks) - at)
            got.append(engine.step([("a", toks[at:at + c], list(range(c)))]))
            at += c
        engine.finish("a")
        close(torch.cat(got).cpu(), ref[:at], 5e-5)


@AB
@pytest.mark.parametrize("dt", [torch.float32, torch.bfloat16], ids=["fp32", "bf16"])
def test_mixed_batches_match_each_request_alone_and_reuse_pages_and_slots(cfg, dt):
    engine, tensors = build(cfg, dtype=dt, max_tokens=256, max_seqs=3)
    prompts = {r: tokens(n, cfg["vocab"], 20 + i) for i, (r, n) in enumerate((("a", 70), ("b", 33), ("c", 5), ("d", 90), ("e", 48)))}
    ref = {r: R.forward(cfg, tensors, t) for r, t in prompts.items()}
    at = {r: 0 for r in prompts}
    got = {r: [] for r in prompts}

    def feed(plan):
        out = engine.step([(r, prompts[r][at[r]:at[r] + c], list(range(c))) for r, c in plan])
        o = 0
        for r, c in plan:
            got[r].append(out[o:o + c])
            o, at[r] = o + c, at[r] + c
            if at[r] == len(prompts[r]):
                engine.finish(r)

    feed([("a", 40), ("b", 2), ("c", 5)])                        # c ends: its slot and page are free again
    feed([("a", 1), ("b", 30), ("d", 17)])                       # d takes c's slot (and must not read c's state)
    feed([("b", 1), ("d", 2), ("a", 1)])                         # b ends
    feed([("e", 1), ("a", 1), ("d", 1)])                         # e starts with a single token in b's slot
    feed([("a", 1), ("e", 30), ("d", 1)])
    feed([("d", 69), ("a", 26), ("e", 2)])                       # a and d end
    feed([("e", 15)])
    for r in prompts:
        assert at[r] == len(prompts[r])
        if dt == torch.float32:
            close(torch.cat(got[r]).cpu(), ref[r], 5e-5)
        else:
            rounding_close(torch.cat(got[r]).cpu(), ref[r], cfg)
    assert engine.free_slots == 3 and engine.free_blocks == 256 // 16


@ALL
def test_logits_do_not_depend_on_the_batch_or_the_cut_beyond_rounding_bf16(cfg):
    engine, _ = build(cfg, dtype=torch.bfloat16)
    a, b = tokens(80, cfg["vocab"], 31), tokens(37, cfg["vocab"], 32)
    alone = whole(engine, "a", a)
    out = engine.step([("b", b[:20], []), ("a", a[:50], list(range(50)))])
    out2 = engine.step([("a", a[50:], list(range(30))), ("b", b[20:], [])])
    engine.release()
    rounding_close(torch.cat([out, out2]).cpu(), alone, cfg)


def test_long_prompt_whole_in_portions_and_decoded_bf16_against_fp32():
    """600 tokens through the tensor-core kernels: the whole prompt, portions beside another request, and single
    tokens agree with the fp32 engine within 16-bit rounding."""
    cfg = CFG_B
    e32, _ = build(cfg, max_tokens=1024, max_seqs=2)
    e16, _ = build(cfg, dtype=torch.bfloat16, max_tokens=1024, max_seqs=2)
    toks = tokens(600, cfg["vocab"], 16)
    want = [0, 100, 255, 256, 300, 400, 511, 512, 550, 590, 599]
    ref = whole(e32, "a", toks, want)
    rounding_close(whole(e16, "a", toks, want), ref)
    got = [e16.step([("b", toks[:100], [0])]), e16.step([("b", toks[100:590], [0, 155, 156, 200, 300, 411, 412, 450]), ("c", toks[:3], [])])]
    got += [e16.step([("b", [t], [0] if i in (0, 9) else [])]) for i, t in enumerate(toks[590:])]
    e16.release()
    rounding_close(torch.cat([g for g in got if g is not None]).cpu(), ref)


def test_greedy_generation_through_the_scheduler():
    cfg = CFG_B
    engine, tensors = build(cfg, max_tokens=256, max_seqs=2)
    prompts = [tokens(n, cfg["vocab"], 40 + i) for i, n in enumerate((9, 30, 3))]     # three requests, two slots
    out = engine.generate(prompts, max_new_tokens=6, prefill_chunk=7, token_budget=12)
    for p, o in zip(prompts, out):
        want = R.greedy(cfg, tensors, p, 6)
        # a near-tie may flip a token in fp32; up to the first difference the texts must agree and it must be a near-tie
        for k, (x, y) in enumerate(zip(o, want)):
            if x != y:
                lg = R.forward(cfg, tensors, p + want[:k])[-1]
                assert abs(lg[x] - lg[y]) < 1e-4
                break
    assert engine.free_slots == 2


def test_registry_serves_a_checkpoint_folder(tmp_path):
    import json

    from dgi_b200 import model_registry, rufedra_layer as Q
    from dgi_b200.ragged_engine import RaggedStepEngine
    from dgi_b200.safetensors_io import write_safetensors

    tensors = Q.random_checkpoint(Q.RufedraConfig.from_dict(CFG_A), seed=5)
    (tmp_path / "config.json").write_text(json.dumps(CFG_A))
    write_safetensors(str(tmp_path / "model.safetensors"), tensors)
    arch, _, shards = model_registry.load_model_dir(str(tmp_path), device=DEV, dtype=torch.float32)
    assert arch.name == "Rufedra" and arch.engine == "ragged"
    engine = RaggedStepEngine(shards, max_tokens=128, max_seqs=1)
    toks = tokens(20, CFG_A["vocab"], 50)
    close(whole(engine, "a", toks), R.forward(CFG_A, tensors, toks), 5e-5)


def test_layer_ranges_as_separate_shards():
    from dgi_b200 import rufedra_layer as Q
    from dgi_b200.ragged_engine import RaggedStepEngine

    cfg = Q.RufedraConfig.from_dict(CFG_A)
    tensors = Q.random_checkpoint(cfg, seed=6)
    shards = Q.build_shards(cfg, tensors, [(0, 2), (2, 3), (3, 6)], DEV, torch.float32)       # the middle one keeps no pages
    engine = RaggedStepEngine(shards, max_tokens=128, max_seqs=2)
    toks = tokens(45, CFG_A["vocab"], 51)
    ref = R.forward(CFG_A, tensors, toks)
    got = [engine.step([("a", toks[:20], list(range(20)))]), engine.step([("a", toks[20:], list(range(25)))])]
    close(torch.cat(got).cpu(), ref, 5e-5)
