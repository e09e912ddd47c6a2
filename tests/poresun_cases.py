"""Small Poresun configurations and inputs for the tests (config.json dictionaries; none of them is a served model's
combination of sizes). Sizes are deliberately unequal where a served model might make them equal or 1. `bias_rows` tells the
synthetic checkpoint how many rows a layer's distance table has (a real checkpoint's tensor shape does)."""
from __future__ import annotations

import torch


def moe(experts=6, top=2, ff=12, shared=10):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    return out


def dense(ff=20, limit=0.8):
    return {"kind": "dense", "ff": ff, "limit": limit}


def _mlp(mlp):
    return dense() if mlp == "dense" else (moe() if mlp == "moe" else mlp)


def att(heads=3, kv_heads=1, dim=8, vdim=6, window=9, scale=0.7, cap=5.0, far=40, rows=12, mlp="dense"):
    mx = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, bias_max=far, bias_rows=rows)
    if window:
        mx["mask"] = dict(size=window)
    if cap:
        mx["softcap"] = cap
    return {"type": "attention", "mixer": mx, "mlp": _mlp(mlp)}


def att2(heads=4, kv_heads=2, dim=6, vdim=10, scale=0.5, temp=(0.4, 7), far=60, rows=10, kv_from=None, window=0, mlp="dense"):
    mx = dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, scale=scale, bias_max=far, bias_rows=rows)
    if temp:
        mx["q_temp"] = dict(coef=temp[0], every=temp[1])
    if kv_from is not None:
        mx["kv_from"] = kv_from
    if window:
        mx["mask"] = dict(size=window)
    return {"type": "attention_2", "mixer": mx, "mlp": _mlp(mlp)}


def lat(heads=3, dim=6, rot=4, vdim=5, rank=14, q_rank=9, scale=0.3, base=500.0, mlp="dense"):
    return {"type": "latent_attention", "mlp": _mlp(mlp),
            "mixer": dict(heads=heads, dim=dim, rot_dim=rot, vdim=vdim, kv_rank=rank, q_rank=q_rank, scale=scale, rot=dict(dims=rot, base=base))}


def config(layers, width=24, vocab=80, eps=1e-5, alpha=1.7, scale=1.4):
    return {"architecture": "Poresun", "vocab": vocab, "width": width, "layers": layers, "norm": {"eps": eps}, "postln_alpha": alpha,
            "embedding": {"scale": scale}}


CASES = {
    "attention_only": config([att(mlp=None), att(heads=4, kv_heads=2, dim=6, vdim=12, window=70, scale=0.5, cap=2.0, far=33, rows=8, mlp=None),
                              att(heads=2, kv_heads=2, dim=10, vdim=4, window=0, cap=0.0, far=128, rows=16, mlp=None)]),
    "attention2_only": config([att2(mlp=None), att2(heads=3, kv_heads=3, dim=5, vdim=8, temp=(1.1, 1), far=9, rows=16, mlp=None),
                               att2(kv_from=0, heads=2, kv_heads=2, dim=6, vdim=10, temp=(0.2, 50), rows=6, mlp=None),
                               att2(heads=8, kv_heads=2, dim=16, vdim=8, temp=None, window=30, mlp=None),
                               att2(kv_from=0, heads=6, kv_heads=2, dim=6, vdim=10, window=12, mlp=None)]),
    "latent_only": config([lat(mlp=None), lat(heads=2, dim=16, rot=8, vdim=12, rank=24, q_rank=20, mlp=None), lat(heads=5, dim=3, rot=2, vdim=7, rank=9, q_rank=5, mlp=None)]),
    "dense": config([att(), att2(mlp=dense(37, 0.3)), lat(mlp=dense(32, 2.0)), att2(kv_from=1, mlp=None), att(heads=2, kv_heads=1, dim=6, vdim=8, window=33, mlp=dense(16, 0.6))],
                    width=40, alpha=0.8),
    "moe": config([att(mlp=moe(experts=8, top=3, ff=10, shared=7)), lat(mlp=moe(experts=3, top=1, ff=20)), att2(mlp=moe(experts=4, top=4, ff=9, shared=0)),
                   att(window=20, mlp=moe(experts=9, top=2, ff=16, shared=16))], width=24),
    "mixed": config([att2(mlp="dense"), att(mlp="moe"), lat(mlp="moe"), att2(kv_from=0, mlp="moe"), att(heads=4, kv_heads=2, dim=6, vdim=9, window=70, mlp=None),
                     lat(heads=4, dim=5, rot=6, vdim=6, mlp=dense(48, 1.1))], width=32, vocab=96, alpha=2.3),
    "odd": config([att(heads=5, kv_heads=5, dim=11, vdim=3, window=129, scale=0.7, cap=30.0, far=77, rows=13, mlp=moe(experts=33, top=5, ff=6, shared=5)),
                   lat(heads=7, dim=5, rot=10, vdim=3, rank=11, q_rank=13, base=20.0, mlp=dense(7, 0.2)),
                   att2(heads=6, kv_heads=2, dim=5, vdim=11, temp=(0.15, 33), far=700, rows=40, mlp=moe(experts=2, top=1, ff=7, shared=33)),
                   att2(heads=2, kv_heads=2, dim=5, vdim=11, kv_from=2, far=5, rows=4, mlp=None)], width=18, vocab=50, eps=1e-6, alpha=1.0, scale=0.4),
    # layers whose weights the tests shape so that one key stands out
    "sharp": config([att(heads=2, kv_heads=1, dim=8, vdim=8, window=100, scale=3.0, cap=40.0, far=150, rows=16, mlp=None)], width=16, vocab=64),
    "sharp2": config([att2(heads=2, kv_heads=1, dim=8, vdim=8, scale=3.0, temp=(0.05, 90), far=150, rows=16, mlp=None),
                      att2(heads=4, kv_heads=1, dim=8, vdim=8, scale=3.0, temp=(0.05, 40), far=90, rows=10, kv_from=0, mlp=None)], width=16, vocab=64),
    "sharp_latent": config([lat(heads=2, dim=8, rot=4, vdim=8, rank=10, q_rank=12, scale=0.5, mlp=None)], width=16, vocab=64),
}


def tokens(n, vocab, seed=0):
    g = torch.Generator().manual_seed(7000 + seed)
    return torch.randint(0, vocab, (n,), generator=g).tolist()


def random_config(seed):
    """A random stack: 2 to 6 layers of the three mixers in any order, head counts and sizes that are and are not multiples of 8, windows
    from 1 token to beyond the prompt and none, distance tables of 2 to 64 rows, layers that read an earlier layer's keys and
    values, dense, routed or no feed-forward."""
    import random

    rng = random.Random(seed)

    def rmlp():
        x = rng.random()
        if x < 0.2:
            return None
        if x < 0.5:
            return dense(rng.choice([8, 20, 37, 64]), rng.choice([0.2, 1.0, 5.0]))
        E = rng.choice([1, 2, 4, 6, 12, 40])
        return moe(experts=E, top=rng.randint(1, min(E, 5)), ff=rng.choice([8, 12, 16, 40, 64]), shared=rng.choice([0, 8, 13, 64]))

    def table():
        rows = rng.choice([2, 4, 8, 10, 16, 32, 64])
        return dict(rows=rows, far=rng.choice([rows // 2 + 1, rows, 4 * rows, 300]))

    layers, owners = [], []
    for i in range(rng.randint(2, 6)):
        x = rng.random()
        G = rng.choice([1, 2, 3])
        if x < 0.35:
            layers.append(att(heads=G * rng.choice([1, 2, 4]), kv_heads=G, dim=rng.choice([3, 6, 8, 16, 20, 32, 72]), vdim=rng.choice([4, 6, 8, 20, 40, 144]),
                              window=rng.choice([0, 1, 2, 7, 31, 64, 65, 100, 400]), scale=rng.uniform(0.05, 0.6), cap=rng.choice([0.0, 1.5, 10.0, 50.0]),
                              mlp=rmlp(), **table()))
        elif x < 0.75:
            if owners and rng.random() < 0.5:
                src = rng.choice(owners)
                o = layers[src]["mixer"]
                geo = dict(heads=o["heads"], kv_heads=o["kv_heads"], dim=o["dim"], vdim=o["vdim"], kv_from=src)
            else:
                geo = dict(heads=G * rng.choice([1, 2, 4]), kv_heads=G, dim=rng.choice([3, 6, 8, 16, 20, 32, 72]), vdim=rng.choice([4, 6, 8, 20, 40, 144]))
                owners.append(i)
            layers.append(att2(scale=rng.uniform(0.05, 0.6), temp=rng.choice([None, (0.3, 1), (0.2, 16), (0.5, 101)]), mlp=rmlp(), **geo, **table()))
        else:
            layers.append(lat(heads=rng.choice([1, 2, 5]), dim=rng.choice([4, 6, 16, 33]), rot=rng.choice([2, 6, 8, 16]), vdim=rng.choice([3, 8, 12, 32]),
                              rank=rng.choice([7, 16, 32, 64]), q_rank=rng.choice([5, 16, 24]), scale=rng.uniform(0.05, 0.4),
                              base=rng.choice([30.0, 10000.0]), mlp=rmlp()))
    return config(layers, width=rng.choice([16, 24, 40, 64, 100, 136]), vocab=rng.choice([50, 96, 200]), eps=rng.choice([1e-6, 1e-5]),
                  alpha=rng.choice([0.5, 1.0, 2.2]), scale=rng.choice([0.5, 1.0, 3.3]))
