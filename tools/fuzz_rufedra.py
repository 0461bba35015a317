"""Random Rufedra configurations (layer orders, head layouts and sizes on and off the tensor-core grid, windows, rotations, branch
weights, convolution taps, states and ranks, missing feed-forwards): the ragged step engine in fp32 and bf16, two requests cut into
random portions and mixed in steps with slots used again, against oracle/rufedra_ref.py.
``python tools/fuzz_rufedra.py [n_seeds] [first]`` on a B200; prints one line per seed and ``bad <count>``."""
import contextlib
import json
import os
import random
import sys
import traceback

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
import torch  # noqa: E402

import dgi_b200  # noqa: E402,F401
from dgi_b200 import rufedra_layer as Q  # noqa: E402
from dgi_b200.ragged_engine import RaggedStepEngine  # noqa: E402
from oracle import rufedra_ref as R  # noqa: E402


def rand_mixer(rng):
    H = rng.choice([1, 2, 3, 4, 6, 8, 12, 20, 40])
    G = rng.choice([g for g in range(1, H + 1) if H % g == 0])
    if rng.random() < 0.5:
        return "delta", {"heads": H, "kv_heads": G, "dim": rng.choice([2, 8, 16, 24, 33, 48, 64, 96, 128, 200, 256]),
                         "vdim": rng.choice([8, 16, 24, 33, 48, 64, 96, 128, 200]), "conv": rng.choice([1, 2, 3, 4, 4, 4, 7])}
    dk = rng.choice([4, 8, 16, 24, 32, 48, 64, 80, 128, 10])
    left = {"heads": H, "kv_heads": G, "dim": dk, "vdim": dk, "scale": rng.choice([0.5, 1.0]) / dk ** 0.5,
            "mask": {"size": rng.choice([1, 2, 7, 16, 31, 32, 33, 40, 64, 100, 1000])},
            "rot": {"base": rng.choice([50.0, 10000.0, 500000.0]), "dims": 2 * rng.randint(0, dk // 2)}}
    right = {"inner": rng.choice([8, 9, 24, 64, 100, 192, 200]), "state": rng.choice([1, 3, 4, 8, 12, 16, 24, 33, 64, 100]),
             "dt_rank": rng.choice([1, 2, 5, 8, 16]), "conv": rng.choice([1, 2, 3, 4, 4, 4, 7])}
    return "parallel", {"left": left, "right": right, "left_scale": rng.choice([1.0, 0.6, -0.5, 0.0]),
                        "right_scale": rng.choice([1.0, 0.9, -0.7, 0.3])}


def rand_cfg(rng):
    layers = []
    for _ in range(rng.randint(1, 6)):
        kind, m = rand_mixer(rng)
        mlp = {"kind": "dense", "ff": rng.choice([8, 24, 33, 64, 200])} if rng.random() < 0.7 else None
        layers.append({"type": kind, "mixer": m, "mlp": mlp})
    return {"architecture": "Rufedra", "width": rng.choice([16, 30, 32, 48, 64, 96, 128, 200]), "vocab": rng.choice([17, 64, 301]),
            "norm": {"eps": rng.choice([1e-6, 1e-5])}, "embedding": {"scale": rng.choice([1.0, 5.5])},
            "logit_scale": rng.choice([0.25, 0.3, 1.0]), "layers": layers}


def row_error(got, ref):
    """The median token's error rms over the reference's rms."""
    return float(((got - ref).pow(2).mean(dim=1).sqrt() / ref.pow(2).mean().sqrt()).median())


@contextlib.contextmanager
def rounded_norms():
    """The oracle with every RMS norm's result rounded to bf16."""
    plain = R.rms
    R.rms = lambda *a: plain(*a).to(torch.bfloat16).to(a[0].dtype)
    try:
        yield
    finally:
        R.rms = plain


def main():
    bad = 0
    first = int(sys.argv[2]) if len(sys.argv) > 2 else 0
    for seed in range(first, first + (int(sys.argv[1]) if len(sys.argv) > 1 else 24)):
        rng = random.Random(seed)
        raw = rand_cfg(rng)
        try:
            cfg = Q.RufedraConfig.from_dict(raw)
            tensors = Q.random_checkpoint(cfg, seed=seed)
            g = torch.Generator().manual_seed(seed)
            n1, n2 = rng.randint(40, 150), rng.randint(1, 60)
            t1 = torch.randint(0, raw["vocab"], (n1,), generator=g).tolist()
            t2 = torch.randint(0, raw["vocab"], (n2,), generator=g).tolist()
            ref1, ref2 = R.forward(raw, tensors, t1), R.forward(raw, tensors, t2)
            # what fp32 arithmetic alone does to this model (the same statement in fp32): the yardstick for the fp32 engine
            cond = max(float((R.forward(raw, tensors, t, dtype=torch.float32).double() - ref).abs().max() / max(1.0, ref.abs().max()))
                       for t, ref in ((t1, ref1), (t2, ref2)))
            # what rounding nothing but the sublayers' inputs to bf16 does to it: the yardstick for the bf16 engine, which
            # rounds projections, activations and cached rows as well
            with rounded_norms():
                cond16 = max(row_error(R.forward(raw, tensors, t), ref) for t, ref in ((t1, ref1), (t2, ref2)))
            for dt, tol in ((torch.float32, max(5e-5, 4.0 * cond)), (torch.bfloat16, max(6e-2, 4.0 * cond16))):
                eng = RaggedStepEngine(Q.build_shards(cfg, tensors, [(0, cfg.num_hidden_layers)], "cuda:0", dt), max_tokens=256,
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
                        # a unit-RMS read-out near zero turns far under rounding: judge the median token
                        err = row_error(gg, ref)
                    if not (err <= tol):
                        bad += 1
                        print("MISMATCH seed", seed, dt, err, "allowed", tol, json.dumps(raw), flush=True)
            print("seed", seed, "ok", [(l["type"][:4], l["mixer"].get("left", l["mixer"])["heads"]) for l in raw["layers"]], flush=True)
        except Exception as e:  # noqa: BLE001
            bad += 1
            print("ERROR seed", seed, type(e).__name__, str(e)[:300], json.dumps(raw), flush=True)
            traceback.print_exc()
    print("bad", bad)
    return bad


if __name__ == "__main__":
    sys.exit(1 if main() else 0)
