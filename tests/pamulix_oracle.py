"""Plain, slow restatement of the Pamulix design in float64 on the CPU, one function per mechanism, written from the design's equations
and sharing nothing with the package: the oracle for tests/test_pamulix*.py.

Notation: x is the residual stream [T, width] of one sequence's tokens at positions 0..T-1; W['name'] are float64 tensors, matrices stored
[out, in].  Every function sees the WHOLE sequence at once (no cache carried between calls): whatever the engine does with pages, portions
and batches must reproduce these numbers."""
import math

import numpy as np
import torch

F = torch.float64


def rms(v, w, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps) * w


def layer_norm(v, w, eps):
    """Weight, no bias."""
    d = v - v.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * w


# ------------------------------------------------------------------ rotation
def pair_frequencies(rot):
    """One frequency per pair, and the amplitude both cosine and sine carry: stretched positions turn the slow pairs `factor` times more
    slowly, leave the fast ones alone, and blend linearly over the pair index in between."""
    n, base, sc = rot["dims"], rot["base"], rot.get("scaling")
    plain = [base ** (-2.0 * i / n) for i in range(n // 2)]
    if not sc:
        return plain, 1.0

    def pair_index(turns):   # the (real-valued) pair that makes this many turns over the original context
        return n * math.log(sc["original"] / (2.0 * math.pi * turns)) / (2.0 * math.log(base))

    lo, hi = max(math.floor(pair_index(sc["fast"])), 0), min(math.ceil(pair_index(sc["slow"])), n - 1)
    out = []
    for i, f in enumerate(plain):
        slow_part = min(max((i - lo) / max(hi - lo, 0.001), 0.0), 1.0)
        out.append(slow_part * f / sc["factor"] + (1.0 - slow_part) * f)
    return out, 1.0 + 0.1 * math.log(sc["factor"])


def rotate(v, rot):
    """v [T, ..., n], row t at position t: neighbours 2i and 2i + 1 of the first rot.dims entries turn together."""
    freq, amp = pair_frequencies(rot)
    out = v.clone()
    p = torch.arange(v.shape[0], dtype=F).view([-1] + [1] * (v.dim() - 2))
    for i, f in enumerate(freq):
        c, s = amp * torch.cos(p * f), amp * torch.sin(p * f)
        a, b = v[..., 2 * i], v[..., 2 * i + 1]
        out[..., 2 * i] = a * c - b * s
        out[..., 2 * i + 1] = b * c + a * s
    return out


# ------------------------------------------------------------------ latent attention
def latent_rows(h, W, p, mx, eps):
    """What a layer caches per position: normed latent row [T, kv_rank], rotated key part shared by the heads [T, rot_dim]."""
    down = h @ W[p + "dkv"].T
    r = mx["kv_rank"]
    return rms(down[:, :r], W[p + "dkv.norm"], eps), rotate(down[:, r:], mx["rot"])


def latent_queries(h, W, p, mx, eps):
    q = (rms(h @ W[p + "dq"].T, W[p + "dq.norm"], eps) @ W[p + "uq"].T).view(h.shape[0], mx["heads"], mx["dim"] + mx["rot_dim"])
    return q[..., :mx["dim"]], rotate(q[..., mx["dim"]:], mx["rot"])


def mixer_latent(h, W, p, mx, eps):
    T, H = h.shape[0], mx["heads"]
    c, kr = latent_rows(h, W, p, mx, eps)
    qn, qr = latent_queries(h, W, p, mx, eps)
    k, v = (c @ W[p + "uk"].T).view(T, H, mx["dim"]), (c @ W[p + "uv"].T).view(T, H, mx["vdim"])
    past = torch.tril(torch.ones(T, T, dtype=torch.bool))
    heads = []
    for a in range(H):
        s = ((qn[:, a] @ k[:, a].T + qr[:, a] @ kr.T) * mx["scale"]).masked_fill(~past, -math.inf)
        heads.append(torch.softmax(s, -1) @ v[:, a])
    return torch.cat(heads, -1) @ W[p + "o"].T


# ------------------------------------------------------------------ chunked attention with a distance bias
def chunk_mask(T, size):
    i = torch.arange(T)
    return (i[None, :] <= i[:, None]) & (i[None, :] // size == i[:, None] // size)


def slope(h, H):
    return 2.0 ** (-8.0 * (h + 1) / H)


def mix_values(v, first, lam):
    return (1.0 - lam) * v + lam * first


def one_more_softmax(s, see):
    """exp(s) over the visible keys divided by (1 + their sum): a key of score 0 without a value."""
    top = torch.clamp(s.masked_fill(~see, -math.inf).amax(-1, keepdim=True), min=0.0)
    e = torch.where(see, torch.exp(s - top), torch.zeros_like(s))
    return e / (torch.exp(-top) + e.sum(-1, keepdim=True))


def mixer_attention(h, W, p, mx, eps, first):
    """first: the values of the first value-mixing layer, [T, G, vdim] (None when this layer is that one, or mixes nothing).
    -> (result, this layer's own values before mixing)"""
    T, H, G = h.shape[0], mx["heads"], mx["kv_heads"]
    q = rms((h @ W[p + "q"].T).view(T, H, mx["dim"]), W[p + "q.norm"], eps)
    k = rms((h @ W[p + "k"].T).view(T, G, mx["dim"]), W[p + "k.norm"], eps)
    own = (h @ W[p + "v"].T).view(T, G, mx["vdim"])
    v = own if first is None else mix_values(own, first, W[p + "vmix"])
    see = chunk_mask(T, mx["mask"]["size"])
    i = torch.arange(T, dtype=F)
    heads = []
    for a in range(H):
        g = a // (H // G)
        s = q[:, a] @ k[:, g].T * mx["scale"] - slope(a, H) * (i[:, None] - i[None, :])
        heads.append(one_more_softmax(s, see) @ v[:, g])
    return torch.cat(heads, -1) @ W[p + "o"].T, own


# ------------------------------------------------------------------ experts
def expert(x, W, p):
    g = x @ W[p + "gate"].T
    return (g * torch.sigmoid(g) * (x @ W[p + "up"].T)) @ W[p + "down"].T


def route(h, W, p, top):
    z = h @ W[p + "router"].T + W[p + "router.b"]
    picked, chosen = torch.topk(z, top, dim=-1)
    return chosen, torch.softmax(picked, -1)


def feed_forward(h, W, p, ml):
    chosen, weight = route(h, W, p, ml["router"]["top"])
    y = torch.zeros_like(h)
    for e in sorted(set(chosen.reshape(-1).tolist())):
        t, k = torch.nonzero(chosen == e, as_tuple=True)
        y.index_add_(0, t, weight[t, k].unsqueeze(-1) * expert(h[t], W, f"{p}e{e}."))
    return y


# ------------------------------------------------------------------ the model
def forward(config, W, tokens, residuals=None):
    """logits [T, vocab] of one sequence; residuals (a list) receives the stream after every layer."""
    eps, m = config["norm"]["eps"], config["residual_mult"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)]
    first = None
    for i, layer in enumerate(config["layers"]):
        p, mx, ml = f"l{i}.", layer["mixer"], layer["mlp"]
        if layer["type"] == "latent_attention":
            y = mixer_latent(x, W, p + "mix.", mx, eps)
        else:
            mixing = mx.get("v_mix", False)
            y, own = mixer_attention(x, W, p + "mix.", mx, eps, first if mixing else None)
            if mixing and first is None:
                first = own
        x = x + m * layer_norm(y, W[p + "norm1"], eps)
        if ml is not None:
            x = x + m * layer_norm(feed_forward(x, W, p + "mlp.", ml), W[p + "norm2"], eps)
        if residuals is not None:
            residuals.append(x)
    return layer_norm(x, W["final.norm"], eps) @ W["head"].T


def greedy(config, W, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(torch.argmax(forward(config, W, ids)[-1])))
    return ids[len(prompt):]


# ------------------------------------------------------------------ small random models
def attention(heads=4, kv_heads=2, dim=12, vdim=10, chunk=20, scale=None, v_mix=True, mlp=None):
    return {"type": "attention", "mlp": mlp, "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "mask": {"size": chunk},
                                                       "scale": scale if scale is not None else dim ** -0.5, "v_mix": v_mix}}


def latent(heads=3, dim=12, rot_dim=8, vdim=10, kv_rank=16, q_rank=14, scale=0.3, base=1000.0, factor=4.0, original=64, fast=8.0, slow=1.0, mlp=None):
    rot = {"base": base, "dims": rot_dim}
    if factor is not None:
        rot["scaling"] = {"factor": factor, "original": original, "fast": fast, "slow": slow}
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank,
                                                              "q_rank": q_rank, "scale": scale, "rot": rot}}


def moe(experts=5, top=2, ff=12):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff}}


def make_config(layers, width=36, vocab=50, eps=1e-5, mult=0.7):
    return {"architecture": "Pamulix", "width": width, "vocab": vocab, "norm": {"eps": eps}, "residual_mult": mult, "layers": layers}


def make_weights(config, seed):
    """-> (float64 weights for this file, bfloat16 tensors for the engine): values exact in bfloat16."""
    g = torch.Generator().manual_seed(seed)
    W = {}
    d, V = config["width"], config["vocab"]

    def put(name, *shape, std=None, mean=0.0):
        std = std if std is not None else 1.0 / math.sqrt(shape[-1])
        W[name] = (torch.randn(*shape, generator=g) * std + mean).to(torch.bfloat16)

    put("embed", V, d, std=1.0)
    for i, layer in enumerate(config["layers"]):
        p, mx, ml = f"l{i}.", layer["mixer"], layer["mlp"]
        H = mx["heads"]
        put(p + "norm1", d, std=0.2, mean=1.0)
        put(p + "mix.o", d, H * mx["vdim"])
        if layer["type"] == "latent_attention":
            r, rq, dr = mx["kv_rank"], mx["q_rank"], mx["rot_dim"]
            put(p + "mix.dq", rq, d)
            put(p + "mix.dq.norm", rq, std=0.2, mean=1.0)
            put(p + "mix.uq", H * (mx["dim"] + dr), rq, std=1.5 / math.sqrt(rq))
            put(p + "mix.dkv", r + dr, d)
            put(p + "mix.dkv.norm", r, std=0.2, mean=1.0)
            put(p + "mix.uk", H * mx["dim"], r)
            put(p + "mix.uv", H * mx["vdim"], r)
        else:
            G = mx["kv_heads"]
            put(p + "mix.q", H * mx["dim"], d)
            put(p + "mix.k", G * mx["dim"], d)
            put(p + "mix.v", G * mx["vdim"], d)
            put(p + "mix.q.norm", mx["dim"], std=0.3, mean=1.2)
            put(p + "mix.k.norm", mx["dim"], std=0.3, mean=1.2)
            if mx.get("v_mix"):
                W[p + "mix.vmix"] = (0.2 + 0.6 * torch.rand((), generator=g)).to(torch.bfloat16)
        if ml is None:
            continue
        put(p + "norm2", d, std=0.2, mean=1.0)
        E = ml["router"]["experts"]
        for e in range(E):
            put(f"{p}mlp.e{e}.gate", ml["expert"]["ff"], d, std=1.5 / math.sqrt(d))
            put(f"{p}mlp.e{e}.up", ml["expert"]["ff"], d, std=1.5 / math.sqrt(d))
            put(f"{p}mlp.e{e}.down", d, ml["expert"]["ff"])
        put(p + "mlp.router", E, d)
        put(p + "mlp.router.b", E, std=0.7)
    put("final.norm", d, std=0.2, mean=1.0)
    put("head", V, d)
    return {k: v.double() for k, v in W.items()}, W


def rel_err(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return float(np.linalg.norm(got - want) / max(np.linalg.norm(want), 1e-30))
