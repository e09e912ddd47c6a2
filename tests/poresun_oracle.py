"""Plain, slow float64 implementation of the Poresun design, one function per mechanism, written from the equations and
sharing no code with the product path. It takes the config.json dictionary and a {name: tensor} dict and processes a whole
sequence at once: no cache, no portions, every row loops over the keys it sees.

The design: x <- n1(alpha x + ls1 * mixer(x)), then x <- n2(alpha x + ls2 * ff(x)), where every n is an RMS norm with a weight
and ls1, ls2 are vectors. Three softmax mixers: "attention" (unit-rms queries and keys, soft-capped scores, a learned bias per
distance bucket, a sliding window), "attention_2" (weighted q / k norms, a query temperature that grows with the position, the
distance bias, optionally another layer's keys and values) and "latent_attention" (query and key/value latents, one rotated
key part for all heads, a sigmoid gate per output channel). The feed-forward is a clamped gated one, or a mixture of
squared-relu experts weighted by the softmax over the chosen logits, plus a shared expert behind a gate. The logits come from the
embedding table.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def bucket(n, rows, far):
    """Row of the bias table for a distance of n positions: one row per distance in the first half of the table, then rows whose
    distances grow geometrically up to `far`; everything beyond shares the last row."""
    half = rows // 2
    if n < half:
        return n
    return min(rows - 1, half + math.floor(math.log(n / half) / math.log(far / half) * (rows - half) + 1e-12))


def distance_bias(rel, far, n_max):
    """rel [B, H] -> [n_max + 1, H]: the bias of every distance."""
    return torch.stack([rel[bucket(n, rel.shape[0], far)] for n in range(n_max + 1)])


def visible(i, size):
    return range(max(0, i - size + 1) if size else 0, i + 1)


def query_temperature(p, qt):
    return 1.0 + float(qt["coef"]) * math.log((p + 1) // int(qt["every"]) + 1)


def softmax_attention(q, k, v, scale, cap=0.0, size=0, bias=None):
    """q [T, H, D], k [T, G, D], v [T, G, DV]: head h uses key/value head h // (H / G). bias [distances, H]: added behind the cap."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for i in range(T):
        js = torch.tensor(visible(i, size))
        kk = k[js].repeat_interleave(H // G, 1)                     # [keys, H, D]
        s = soft_cap(torch.einsum("jhd,hd->jh", kk, q[i]) * scale, cap)
        if bias is not None:
            s = s + bias[i - js]
        out[i] = torch.einsum("jh,jhv->hv", torch.softmax(s, 0), v[js].repeat_interleave(H // G, 1))
    return out


def rotate_pairs(x, base):
    """x [T, heads, dims]: channels 2i and 2i + 1 turn together by position * base^(-2i / dims)."""
    T, _, n = x.shape
    f = torch.tensor([base ** (-2.0 * i / n) for i in range(n // 2)], dtype=F64)
    a = torch.arange(T, dtype=F64)[:, None] * f
    c, s = torch.cos(a)[:, None], torch.sin(a)[:, None]
    u, v = x[..., 0::2], x[..., 1::2]
    return torch.stack([u * c - v * s, v * c + u * s], -1).flatten(-2)


def attention_mixer(h, cfg, t, p, eps, weighted, kv=None, leave_out=()):
    """Both attention mixers (weighted: q / k norms with a weight). kv: another layer's (keys, values). Returns (output, (k, v))."""
    H, G, D = int(cfg["heads"]), int(cfg["kv_heads"]), int(cfg["dim"])
    DV = int(cfg.get("vdim", D))
    T = h.shape[0]
    q = rms((h @ t[p + "q"].T).view(T, H, D), eps)
    if weighted:
        q = q * t[p + "q.norm"]
    if cfg.get("q_temp") and "q_temp" not in leave_out:
        q = q * torch.tensor([query_temperature(i, cfg["q_temp"]) for i in range(T)], dtype=F64)[:, None, None]
    if kv is None:
        k = rms((h @ t[p + "k"].T).view(T, G, D), eps)
        if weighted:
            k = k * t[p + "k.norm"]
        kv = (k, (h @ t[p + "v"].T).view(T, G, DV))
    bias = None if "bias" in leave_out else distance_bias(t[p + "rel"], float(cfg["bias_max"]), T)
    size = 0 if "window" in leave_out else int((cfg.get("mask") or {}).get("size") or 0)
    cap = 0.0 if "softcap" in leave_out else float(cfg.get("softcap") or 0.0)
    o = softmax_attention(q, kv[0], kv[1], float(cfg["scale"]), cap, size, bias)
    return o.reshape(T, H * DV) @ t[p + "o"].T, kv


def latent_mixer(h, cfg, t, p, eps, leave_out=()):
    H, D, R, rank = int(cfg["heads"]), int(cfg["dim"]), int(cfg["rot_dim"]), int(cfg["kv_rank"])
    DV, base = int(cfg["vdim"]), float(cfg["rot"]["base"])
    T = h.shape[0]
    cq = rms(h @ t[p + "dq"].T, eps) * t[p + "dq.norm"]
    q = (cq @ t[p + "uq"].T).view(T, H, D + R)
    kv = h @ t[p + "dkv"].T
    c = rms(kv[:, :rank], eps) * t[p + "dkv.norm"]
    turn = (lambda x: x) if "rotation" in leave_out else (lambda x: rotate_pairs(x, base))
    kr = turn(kv[:, None, rank:]).expand(T, H, R)
    k = torch.cat([(c @ t[p + "uk"].T).view(T, H, D), kr], -1)
    q = torch.cat([q[..., :D], turn(q[..., D:])], -1)
    o = softmax_attention(q, k, (c @ t[p + "uv"].T).view(T, H, DV), float(cfg["scale"])).reshape(T, H * DV)
    if "gate" not in leave_out:
        o = o * torch.sigmoid(h @ t[p + "g"].T)
    return o @ t[p + "o"].T


def clamped_glu(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1.0)


def dense_ff(h, t, p, limit):
    return clamped_glu(h @ t[p + "gate"].T, h @ t[p + "up"].T, limit) @ t[p + "down"].T


def expert(h, t, p):
    return torch.clamp(h @ t[p + "up"].T, min=0.0).pow(2) @ t[p + "down"].T


def route(z, top):
    """z [E] logits (bias included): (the `top` largest in descending order, the softmax over them)."""
    order = torch.sort(z, descending=True, stable=True).indices[:top]
    return order.tolist(), torch.softmax(z[order], 0)


def routed_ff(h, mlp, t, p, leave_out=()):
    z = h @ t[p + "router"].T + (0.0 if "router_bias" in leave_out else t[p + "router.b"])
    top = int(mlp["router"]["top"])
    out = torch.zeros_like(h)
    for i in range(h.shape[0]):
        for e, w in zip(*route(z[i], top)):
            out[i] += w * expert(h[i:i + 1], t, f"{p}e{e}.")[0]
    if mlp.get("shared") and "shared" not in leave_out:
        g = 1.0 if "shared_gate" in leave_out else torch.sigmoid(h @ t[p + "shared.sg"].T)
        out = out + g * expert(h, t, p + "shared.")
    return out


def forward(cfg, tensors, ids, layer_outputs=False, leave_out=()):
    """Logits [T, vocab] of one sequence (and, with layer_outputs, the residual stream after every layer). leave_out names
    mechanisms to drop ("bias", "softcap", "window", "q_temp",
    "rotation", "gate", "router_bias", "shared", "shared_gate", "layer_scale", "alpha"): tests use it to show that their weights
    would expose a product that dropped one."""
    t = {k: v.to(F64) for k, v in tensors.items()}
    eps, alpha = float(cfg["norm"]["eps"]), float(cfg.get("postln_alpha", 1.0))
    if "alpha" in leave_out:
        alpha = 1.0
    x = t["embed"][torch.as_tensor(ids, dtype=torch.long)] * float((cfg.get("embedding") or {}).get("scale", 1.0))
    outs, caches = [], {}
    for i, L in enumerate(cfg["layers"]):
        p, mx = f"l{i}.", L["mixer"]
        if L["type"] == "latent_attention":
            y = latent_mixer(x, mx, t, p + "mix.", eps, leave_out)
        elif L["type"] in ("attention", "attention_2"):
            src = mx.get("kv_from")
            y, caches[i] = attention_mixer(x, mx, t, p + "mix.", eps, L["type"] == "attention_2", None if src is None else caches[int(src)], leave_out)
        else:
            raise NotImplementedError(L["type"])
        ls = (lambda n: 1.0) if "layer_scale" in leave_out else (lambda n: t[p + n])
        x = rms(alpha * x + ls("ls1") * y, eps) * t[p + "norm1"]
        mlp = L.get("mlp")
        if mlp is not None:
            y = dense_ff(x, t, p + "mlp.", float(mlp["limit"])) if mlp["kind"] == "dense" else routed_ff(x, mlp, t, p + "mlp.", leave_out)
            x = rms(alpha * x + ls("ls2") * y, eps) * t[p + "norm2"]
        outs.append(x)
    logits = (rms(x, eps) * t["final.norm"]) @ t["embed"].T
    return (logits, torch.stack(outs)) if layer_outputs else logits


def greedy(cfg, tensors, prompt, n_new):
    """The n_new tokens that greedy decoding appends to the prompt (the whole sequence is recomputed for every token)."""
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(forward(cfg, tensors, ids)[-1].argmax()))
    return ids[len(prompt):]
