"""Random Zuderax configurations (layer orders, layers that run another layer's weights, head layouts and sizes on and off
the tensor-core grid, latent ranks, windows, gate caps, state groups, norm parts, convolution taps, expert groups, dense and
missing feed-forwards): the ragged step engine in fp32 and bf16, two requests cut into random portions and mixed in steps with
slots used again, against oracle/zuderax_ref.py.
``python tools/fuzz_zuderax.py [n_seeds] [first]`` on a B200; prints one line per seed and ``bad <count>``."""
import contextlib
import json
import os
import random
import sys
import traceback

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
import torch  # noqa: E402

import dgi_b200  # noqa: E402,F401
from dgi_b200 import zuderax_layer as Z  # noqa: E402
from dgi_b200.ragged_engine import RaggedStepEngine  # noqa: E402
from oracle import zuderax_ref as R  # noqa: E402


def rand_mlp(rng):
    kind = rng.random()
    if kind < 0.15:
        return None
    if kind < 0.45:
        return {"kind": "dense", "ff": rng.choice([8, 24, 33, 64, 200])}
    groups = rng.choice([1, 1, 2, 3, 4])
    E = groups * rng.choice([1, 2, 3, 4, 8])
    keep = rng.randint(1, groups)
    top = rng.randint(1, min(keep * (E // groups), 5))
    mlp = {"kind": "moe", "expert": {"ff": rng.choice([8, 24, 40, 64, 136])},
           "router": {"experts": E, "top": top, "scale": rng.choice([0.5, 1.0, 2.5]), "groups": {"count": groups, "keep": keep}}}
    if rng.random() < 0.7:
        mlp["shared"] = {"ff": rng.choice([8, 20, 64, 96])}
    return mlp


def rand_mixer(rng):
    kind = rng.choice(["latent_attention", "mlstm", "mamba2"])
    H = rng.choice([1, 2, 3, 4, 6, 8, 12])
    if kind == "latent_attention":
        H = rng.choice([H, 16, 20, 33])
        dn, dr = rng.choice([2, 4, 8, 16, 24, 32, 64, 96]), rng.choice([2, 4, 8, 16, 32, 64])
        rank = rng.choice([4, 8, 24, 32, 48, 56, 64, 96, 128, 192, 256, 2 * rng.randint(2, 60)])
        m = {"heads": H, "dim": dn, "rot_dim": dr, "vdim": rng.choice([2, 8, 16, 24, 32, 64, 100]), "kv_rank": rank,
             "scale": rng.choice([0.5, 1.0]) / (dn + dr) ** 0.5, "mask": {"size": rng.choice([1, 2, 7, 16, 31, 32, 33, 40, 64, 100, 1000])},
             "rot": {"base": rng.choice([50.0, 10000.0, 500000.0]), "dims": dr}}
    elif kind == "mlstm":
        m = {"heads": H, "dim": rng.choice([2, 8, 16, 24, 33, 48, 64, 96, 128, 200, 256]),
             "vdim": rng.choice([8, 16, 24, 33, 48, 64, 96, 128, 200]), "gate_cap": rng.choice([2.0, 5.0, 15.0, 30.0])}
    else:
        dv = rng.choice([4, 8, 16, 24, 32, 48, 64, 100])
        m = {"heads": H, "vdim": dv, "state": rng.choice([1, 4, 8, 16, 24, 33, 48, 64, 100, 128, 200]),
             "groups": rng.choice([g for g in range(1, H + 1) if H % g == 0]), "conv": rng.choice([1, 2, 3, 4, 4, 4, 7]),
             "norm_groups": rng.choice([g for g in range(1, H * dv + 1) if (H * dv) % g == 0 and H * dv // g >= 4])}
    return kind, m


def rand_cfg(rng):
    layers = []
    for _ in range(rng.randint(1, 6)):
        owners = [i for i, layer in enumerate(layers) if "weights_of" not in layer]
        if owners and rng.random() < 0.2:
            j = rng.choice(owners)
            layers.append(dict(layers[j], weights_of=j))
        else:
            kind, m = rand_mixer(rng)
            layers.append({"type": kind, "mixer": m, "mlp": rand_mlp(rng)})
    return {"architecture": "Zuderax", "width": rng.choice([16, 30, 32, 48, 64, 96, 128, 200]), "vocab": rng.choice([17, 64, 301]),
            "norm": {"eps": rng.choice([1e-6, 1e-5])}, "logit_scale": rng.choice([0.25, 0.3, 1.0]), "layers": layers}


def row_error(got, ref):
    """The median token's error rms over the reference's rms."""
    return float(((got - ref).pow(2).mean(dim=1).sqrt() / ref.pow(2).mean().sqrt()).median())


@contextlib.contextmanager
def rounded_norms():
    """The oracle with every norm's output rounded to bf16."""
    plain = R.dyn_tanh
    R.dyn_tanh = lambda *a: plain(*a).to(torch.bfloat16).to(a[0].dtype)
    try:
        yield
    finally:
        R.dyn_tanh = plain


def main():
    bad = 0
    first = int(sys.argv[2]) if len(sys.argv) > 2 else 0
    for seed in range(first, first + (int(sys.argv[1]) if len(sys.argv) > 1 else 24)):
        rng = random.Random(seed)
        raw = rand_cfg(rng)
        try:
            cfg = Z.ZuderaxConfig.from_dict(raw)
            tensors = Z.random_checkpoint(cfg, seed=seed)
            g = torch.Generator().manual_seed(seed)
            n1, n2 = rng.randint(40, 150), rng.randint(1, 60)
            t1 = torch.randint(0, raw["vocab"], (n1,), generator=g).tolist()
            t2 = torch.randint(0, raw["vocab"], (n2,), generator=g).tolist()
            ref1, ref2 = R.forward(raw, tensors, t1), R.forward(raw, tensors, t2)
            # what fp32 arithmetic alone does to this model (the same statement in fp32): the yardstick for the fp32 engine
            cond = max(float((R.forward(raw, tensors, t, dtype=torch.float32).double() - ref).abs().max() / max(1.0, ref.abs().max()))
                       for t, ref in ((t1, ref1), (t2, ref2)))
            # what rounding nothing but the sublayers' inputs to bf16 does to it: the yardstick for the bf16 engine, which
            # rounds projections, activations and cached rows as well (and flips a routing near-tie here and there, whose
            # token the recurrent state then carries on)
            with rounded_norms():
                cond16 = max(row_error(R.forward(raw, tensors, t), ref) for t, ref in ((t1, ref1), (t2, ref2)))
            for dt, tol in ((torch.float32, max(5e-5, 4.0 * cond)), (torch.bfloat16, max(6e-2, 4.0 * cond16))):
                eng = RaggedStepEngine(Z.build_shards(cfg, tensors, [(0, cfg.num_hidden_layers)], "cuda:0", dt), max_tokens=256,
                                       max_seqs=2)
                eng.step([("z", t2[:7], [])])        # a request that leaves: its slot and page are used again
                eng.finish("z")
                got1, got2, a1, a2 = [], [], 0, 0
                while a1 < n1 or a2 < n2:
                    entries = []
                    c1 = min(n1 - a1, rng.choice([1, 1, 2, 3, 17, 40]))
                    c2 = min(n2 - a2, rng.choice([0, 1, 2, 9]))
                    if c1:
                        entries.append(("a", t1[a1:a1 + c1], list(range(c1))))
                    if c2:
                        entries.append(("b", t2[a2:a2 + c2], list(range(c2))))
                    if rng.random() < 0.5:
                        entries.reverse()
                    if not entries:
                        continue
                    out, o = eng.step(entries), 0
                    for rid, toks, _ in entries:
                        (got1 if rid == "a" else got2).append(out[o:o + len(toks)])
                        o += len(toks)
                    a1 += c1
                    a2 += c2
                eng.release()
                for got, ref in ((got1, ref1), (got2, ref2)):
                    gg = torch.cat(got).cpu().double()
                    if dt == torch.float32:
                        err = float((gg - ref).abs().max() / max(1.0, ref.abs().max()))
                    else:
                        # a routing near-tie that 16-bit rounding flips changes a token's whole feed-forward output: judge
                        # the median token
                        err = row_error(gg, ref)
                    if not (err <= tol):
                        bad += 1
                        print("MISMATCH seed", seed, dt, err, "allowed", tol, json.dumps(raw), flush=True)
            print("seed", seed, "ok", [(l["type"][:4], l["mixer"]["heads"], l["mixer"]["vdim"]) for l in raw["layers"]], flush=True)
        except Exception as e:  # noqa: BLE001
            bad += 1
            print("ERROR seed", seed, type(e).__name__, str(e)[:300], json.dumps(raw), flush=True)
            traceback.print_exc()
    print("bad", bad)
    return bad


if __name__ == "__main__":
    sys.exit(1 if main() else 0)
