"""Small Kapitar configurations and inputs for the tests (config.json dictionaries; none of them is a served model's
combination of sizes). Sizes are deliberately unequal where a served model might make them equal or 1."""
from __future__ import annotations

import torch


def moe(experts=6, top=2, ff=12, groups=(3, 2), shared=10):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if groups:
        out["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def dense(ff=20):
    return {"kind": "dense", "ff": ff}


def _mlp(mlp):
    return dense() if mlp == "dense" else (moe() if mlp == "moe" else mlp)


def att(heads=3, kv_heads=1, dim=8, vdim=6, window=9, keep=3, scale=0.3, cap=5.0, diff=0.3, mlp="dense"):
    mx = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, diff=diff)
    if window:
        mx["mask"] = dict(size=window)
        if keep:
            mx["mask"]["keep_first"] = keep
    if cap:
        mx["softcap"] = cap
    return {"type": "attention", "mixer": mx, "mlp": _mlp(mlp)}


def light(heads=2, dim=6, vdim=10, decay=None, mlp="dense"):
    decay = decay if decay is not None else [0.55, 0.9, 0.97, 0.999, 0.8, 1.0][:heads]
    return {"type": "lightning", "mixer": dict(heads=heads, dim=dim, vdim=vdim, decay=decay), "mlp": _mlp(mlp)}


def config(layers, width=24, vocab=80, eps=1e-5):
    return {"architecture": "Kapitar", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}}


CASES = {
    "attention_only": config([att(mlp=None), att(heads=4, kv_heads=2, dim=6, vdim=12, window=70, keep=5, scale=0.5, diff=0.7, mlp=None),
                              att(heads=2, kv_heads=2, dim=10, vdim=4, window=0, cap=2.0, diff=0.0, mlp=None),
                              att(heads=1, kv_heads=1, dim=4, vdim=7, window=5, keep=0, cap=0.0, mlp=None)]),
    "lightning_only": config([light(mlp=None), light(heads=4, dim=9, vdim=5, mlp=None), light(heads=1, dim=20, vdim=20, decay=[1.0], mlp=None)]),
    "dense": config([att(), light(), att(heads=2, kv_heads=1, dim=6, vdim=8, window=33, keep=17, mlp=dense(37)), light(heads=3, dim=4, vdim=4, mlp=None)],
                    width=40),
    "moe": config([att(mlp=moe(experts=8, top=3, ff=10, groups=(4, 2), shared=7)), light(mlp=moe(experts=3, top=1, ff=20, groups=None)),
                   att(window=20, keep=1, mlp=moe(experts=4, top=4, ff=9, groups=(4, 4), shared=0)),
                   light(mlp=moe(experts=9, top=2, ff=16, groups=(3, 1), shared=16))], width=24),
    "mixed": config([att(mlp="dense"), light(mlp="moe"), att(heads=4, kv_heads=2, dim=6, vdim=9, window=70, keep=10, mlp="moe"), att(mlp=None),
                     light(heads=3, dim=12, vdim=4, mlp="dense")], width=32, vocab=96),
    "odd": config([att(heads=5, kv_heads=5, dim=11, vdim=3, window=129, keep=66, scale=0.7, cap=30.0, mlp=moe(experts=33, top=5, ff=6, groups=(11, 7), shared=5)),
                   light(heads=5, dim=17, vdim=3, mlp=dense(7)),
                   att(heads=6, kv_heads=2, dim=5, vdim=11, window=2, keep=1, mlp=moe(experts=2, top=1, ff=7, groups=(1, 1), shared=33)),
                   light(heads=1, dim=40, vdim=33, decay=[0.0], mlp=None)], width=18, vocab=50, eps=1e-6),
    # one attention layer whose weights the tests shape so that one key stands out
    "sharp": config([att(heads=2, kv_heads=1, dim=8, vdim=8, window=100, keep=6, scale=0.5, cap=40.0, diff=0.4, mlp=None)], width=16, vocab=64),
}


def tokens(n, vocab, seed=0):
    g = torch.Generator().manual_seed(5000 + seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def random_config(seed):
    """A random stack: 2 to 6 layers of the two mixers in any order, head counts and sizes that are and are not multiples of 8,
    windows from 1 token to beyond the prompt with 0 to 80 kept positions and none at all, dense, routed or no feed-forward."""
    import random

    rng = random.Random(seed)

    def rmlp():
        x = rng.random()
        if x < 0.2:
            return None
        if x < 0.5:
            return dense(rng.choice([8, 20, 37, 64]))
        E = rng.choice([1, 2, 4, 6, 8, 12, 18, 40])
        count = rng.choice([c for c in range(1, E + 1) if E % c == 0])
        keep = rng.randint(1, count)
        top = rng.randint(1, min(keep * (E // count), 5))
        return moe(experts=E, top=top, ff=rng.choice([8, 12, 16, 40, 64]), groups=None if rng.random() < 0.2 else (count, keep),
                   shared=rng.choice([0, 8, 13, 64]))

    layers = []
    for _ in range(rng.randint(2, 6)):
        if rng.random() < 0.6:
            G = rng.choice([1, 2, 3])
            layers.append(att(heads=G * rng.choice([1, 2, 4]), kv_heads=G, dim=rng.choice([3, 6, 8, 16, 20, 32, 72]), vdim=rng.choice([4, 6, 8, 20, 40, 144]),
                              window=rng.choice([0, 1, 2, 7, 31, 64, 65, 100, 400]), keep=rng.choice([0, 1, 4, 20, 64, 80]), scale=rng.uniform(0.05, 0.5),
                              cap=rng.choice([0.0, 1.5, 10.0, 50.0]), diff=rng.uniform(0.0, 0.8), mlp=rmlp()))
        else:
            H = rng.choice([1, 2, 5])
            layers.append(light(heads=H, dim=rng.choice([4, 6, 16, 20, 33]), vdim=rng.choice([3, 8, 12, 17]),
                                decay=[rng.choice([0.3, 0.6, 0.9, 0.98, 0.999, 1.0]) for _ in range(H)], mlp=rmlp()))
    return config(layers, width=rng.choice([16, 24, 40, 64, 100, 136]), vocab=rng.choice([50, 96, 200]), eps=rng.choice([1e-6, 1e-5]))
