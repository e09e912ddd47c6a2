"""Plain, slow float64 implementation of the Kapitar design, one function per mechanism, written from the equations and
sharing no code with the product path. It takes the config.json dictionary and a {name: tensor} dict and processes a whole
sequence at once: no cache, no carried state, every row loops over the keys it sees and every recurrence over its tokens.

The design: x <- x + n1b(mixer(n1(x))), then x <- x + n2b(ff(n2(x))), where every n is a layer norm with a weight and no bias.
The mixer is differential attention ("attention": two softmax maps per head over the same values, soft-capped scores, a
sliding window that keeps the first tokens, no positions) or linear attention with one fixed decay per head ("lightning":
silu on queries, keys and values, one norm over all heads, a sigmoid gate). The feed-forward is two matrices around a squared
relu, or a mixture of gelu experts with a sigmoid router limited to the best groups of experts, plus a shared expert. The
logits come from the embedding table.
"""
from __future__ import annotations

import math

import torch

F64 = torch.float64


def layer_norm(x, w, eps):
    """(x - mean) / sqrt(mean squared deviation + eps) * w over the last axis."""
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt(d.pow(2).mean(-1, keepdim=True) + eps) * w


def rms(x, eps):
    return x / torch.sqrt(x.pow(2).mean(-1, keepdim=True) + eps)


def silu(z):
    return z * torch.sigmoid(z)


def gelu_erf(z):
    return 0.5 * z * (1.0 + torch.erf(z / math.sqrt(2.0)))


def relu2(z):
    return torch.clamp(z, min=0.0).pow(2)


def soft_cap(s, cap):
    return cap * torch.tanh(s / cap) if cap else s


def visible(i, size, keep_first):
    """Positions that position i sees: itself and earlier ones, within `size` positions (0: all) or among the first `keep_first`."""
    return [j for j in range(i + 1) if size <= 0 or i - j < size or j < keep_first]


def softmax_map(q, k, v, scale, cap, size, keep_first):
    """One attention map. q [T, H, D], k [T, G, D], v [T, G, DV]: head h uses key/value head h // (H / G)."""
    T, H, _ = q.shape
    G = k.shape[1]
    out = torch.zeros(T, H, v.shape[-1], dtype=F64)
    for i in range(T):
        js = torch.tensor(visible(i, size, keep_first))
        for h in range(H):
            g = h // (H // G)
            w = torch.softmax(soft_cap((k[js, g] @ q[i, h]) * scale, cap), 0)
            out[i, h] = w @ v[js, g]
    return out


def diff_lambda(t, p, diff):
    """The layer's weight of the second map."""
    return torch.exp((t[p + "lq1"] * t[p + "lk1"]).sum()) - torch.exp((t[p + "lq2"] * t[p + "lk2"]).sum()) + diff


def diff_combine(a1, a2, lam, diff, eps):
    """Difference of the two maps, each head brought to unit rms, times what the second map's starting weight leaves."""
    return rms(a1 - lam * a2, eps) * (1.0 - diff)


def attention_mixer(h, cfg, t, p, eps, leave_out=()):
    H, G, D, DV = int(cfg["heads"]), int(cfg["kv_heads"]), int(cfg["dim"]), int(cfg["vdim"])
    T = h.shape[0]
    b = (lambda n: 0.0) if "bias" in leave_out else (lambda n: t[p + n + ".b"])
    q = (h @ t[p + "q"].T + b("q")).view(T, H, 2, D)
    k = (h @ t[p + "k"].T + b("k")).view(T, G, 2, D)
    v = (h @ t[p + "v"].T + b("v")).view(T, G, DV)
    cap = 0.0 if "softcap" in leave_out else float(cfg.get("softcap") or 0.0)
    mask = cfg.get("mask") or {}
    size = 0 if "window" in leave_out else int(mask.get("size", 0))
    keep = 0 if "keep_first" in leave_out else int(mask.get("keep_first", 0))
    a = [softmax_map(q[:, :, m], k[:, :, m], v, float(cfg["scale"]), cap, size, keep) for m in range(2)]
    diff = float(cfg["diff"])
    lam = 0.0 if "second_map" in leave_out else diff_lambda(t, p, diff)
    return diff_combine(a[0], a[1], lam, diff, eps).reshape(T, H * DV) @ t[p + "o"].T


def decayed_sum(q, k, v, decay):
    """One head. q, k [T, N], v [T, P]: S <- decay S + k_t v_t^T, o_t = S^T q_t (the read-out sees the token's own write)."""
    S = torch.zeros(k.shape[1], v.shape[1], dtype=F64)
    out = torch.zeros_like(v)
    for i in range(k.shape[0]):
        S = decay * S + torch.outer(k[i], v[i])
        out[i] = S.T @ q[i]
    return out


def lightning_mixer(h, cfg, t, p, eps):
    H, N, P = int(cfg["heads"]), int(cfg["dim"]), int(cfg["vdim"])
    T = h.shape[0]
    q, k = silu(h @ t[p + "q"].T).view(T, H, N), silu(h @ t[p + "k"].T).view(T, H, N)
    v = silu(h @ t[p + "v"].T).view(T, H, P)
    o = torch.stack([decayed_sum(q[:, i], k[:, i], v[:, i], float(cfg["decay"][i])) for i in range(H)], 1).reshape(T, H * P)
    o = rms(o, eps) * t[p + "norm"]                                # one norm over all heads together
    return (o * torch.sigmoid(h @ t[p + "g"].T)) @ t[p + "o"].T


def dense_ff(h, t, p):
    return relu2(h @ t[p + "up"].T) @ t[p + "down"].T


def expert(h, t, p):
    return gelu_erf(h @ t[p + "up"].T) @ t[p + "down"].T


def route_scores(s, router, group_top=2):
    """s [E] scores of one row: (chosen experts in descending order, their scores). Groups of neighbours score as the sum of
    their two largest scores; experts outside the best groups.keep groups cannot be chosen."""
    E, top, gr = s.shape[0], int(router["top"]), router.get("groups")
    allowed = torch.ones(E, dtype=torch.bool)
    if gr:
        per = E // int(gr["count"])
        gs = torch.stack([torch.sort(s[g * per:(g + 1) * per], descending=True).values[:group_top].sum() for g in range(int(gr["count"]))])
        kept = torch.sort(gs, descending=True, stable=True).indices[:int(gr["keep"])].tolist()
        allowed = torch.tensor([e // per in kept for e in range(E)])
    order = torch.sort(torch.where(allowed, s, torch.full_like(s, -1.0)), descending=True, stable=True).indices[:top]
    return order.tolist(), s[order]


def routed_ff(h, mlp, t, p, leave_out=()):
    r = dict(mlp["router"])
    if "groups" in leave_out:
        r.pop("groups", None)
    s = torch.sigmoid(h @ t[p + "router"].T)
    out = torch.zeros(h.shape[0], t[p + "e0.down"].shape[0], dtype=F64)
    for i in range(h.shape[0]):
        idx, w = route_scores(s[i], r, 1 if "group_sum" in leave_out else 2)
        for e, we in zip(idx, w):
            out[i] += we * expert(h[i:i + 1], t, f"{p}e{e}.")[0]
    if mlp.get("shared") and "shared" not in leave_out:
        out = out + expert(h, t, p + "shared.")
    return out


def forward(cfg, tensors, ids, layer_outputs=False, leave_out=()):
    """Logits [T, vocab] of one sequence (and, with layer_outputs, the residual stream after every layer). leave_out names
    mechanisms to drop ("bias", "softcap", "window", "keep_first", "second_map", "groups", "group_sum" (a group scores as its best
    expert alone), "shared"): tests use it to show that their weights would expose a product that dropped one."""
    t = {k: v.to(F64) for k, v in tensors.items()}
    eps = float(cfg["norm"]["eps"])
    x = t["embed"][torch.as_tensor(ids, dtype=torch.long)]
    outs = []
    for i, L in enumerate(cfg["layers"]):
        p = f"l{i}."
        h = layer_norm(x, t[p + "norm1"], eps)
        if L["type"] == "attention":
            y = attention_mixer(h, L["mixer"], t, p + "mix.", eps, leave_out)
        elif L["type"] == "lightning":
            y = lightning_mixer(h, L["mixer"], t, p + "mix.", eps)
        else:
            raise NotImplementedError(L["type"])
        x = x + layer_norm(y, t[p + "norm1b"], eps)
        mlp = L.get("mlp")
        if mlp is not None:
            h = layer_norm(x, t[p + "norm2"], eps)
            y = dense_ff(h, t, p + "mlp.") if mlp["kind"] == "dense" else routed_ff(h, mlp, t, p + "mlp.", leave_out)
            x = x + layer_norm(y, t[p + "norm2b"], eps)
        outs.append(x)
    logits = layer_norm(x, t["final.norm"], eps) @ t["embed"].T
    return (logits, torch.stack(outs)) if layer_outputs else logits


def greedy(cfg, tensors, prompt, n_new):
    """The n_new tokens that greedy decoding appends to the prompt (the whole sequence is recomputed for every token)."""
    ids = list(prompt)
    for _ in range(n_new):
        ids.append(int(forward(cfg, tensors, ids)[-1].argmax()))
    return ids[len(prompt):]
