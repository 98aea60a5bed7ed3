"""Plain, slow restatement of the Zasapel design in float64 on the CPU, one function per mechanism, written from the design's equations
and sharing nothing with the package: the oracle for tests/test_zasapel*.py.

Notation: x is the residual stream [T, width] of one sequence's tokens at positions 0..T-1; W['name'] are float64 tensors, matrices stored
[out, in].  Every function sees the WHOLE sequence at once (no cache carried between calls): whatever the engine does with pages, slots,
portions and batches must reproduce these numbers."""
import math

import numpy as np
import torch

F = torch.float64


def rms_unit(v, eps):
    return v / torch.sqrt((v * v).mean(-1, keepdim=True) + eps)


def norm_around_zero(v, w, eps):
    """RMS norm whose stored weight is the distance from one."""
    return rms_unit(v, eps) * (1.0 + w)


def position_vector(T, width):
    """Interleaved sines and cosines: entry c has the frequency of the pair it belongs to."""
    out = torch.zeros(T, width, dtype=F)
    p = torch.arange(T, dtype=F)
    for c in range(width):
        a = p * 10000.0 ** (-2.0 * (c // 2) / width)
        out[:, c] = torch.cos(a) if c % 2 else torch.sin(a)
    return out


def with_conv(x, taps_w):
    """x + its causal convolution over time, channel by channel; the last tap is the token's own."""
    width, taps = taps_w.shape
    out = x.clone()
    for t in range(x.shape[0]):
        for j in range(taps):
            s = t - taps + 1 + j
            if s >= 0:
                out[t] += taps_w[:, j] * x[s]
    return out


def mixer_mingru(h, W, p):
    z = torch.sigmoid(h @ W[p + "z"].T + W[p + "z.b"])
    u = h @ W[p + "x"].T + W[p + "x.b"]
    cand = torch.where(u >= 0, u + 0.5, torch.sigmoid(u))
    g = h @ W[p + "g"].T
    S = torch.zeros_like(z[0])
    rows = []
    for t in range(h.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * cand[t]
        rows.append(S * g[t] * torch.sigmoid(g[t]))
    return torch.stack(rows) @ W[p + "o"].T


def latent_rows(h, W, p, eps):
    """What a layer caches per position."""
    return rms_unit(h @ W[p + "dkv"].T, eps) * W[p + "dkv.norm"]


def latent_queries(h, W, p, mx, eps):
    c_q = rms_unit(h @ W[p + "dq"].T, eps) * W[p + "dq.norm"]
    return (c_q @ W[p + "uq"].T).view(h.shape[0], mx["heads"], mx["dim"])


def mixer_latent(h, W, p, mx, eps, c):
    """c = the latent rows of this layer or of the layer it borrows from."""
    T, H = h.shape[0], mx["heads"]
    q = latent_queries(h, W, p, mx, eps)
    k = (c @ W[p + "uk"].T).view(T, H, mx["dim"])
    v = (c @ W[p + "uv"].T).view(T, H, mx["vdim"])
    past = torch.tril(torch.ones(T, T, dtype=torch.bool))
    gate = torch.sigmoid(h @ W[p + "g"].T)          # one number per head
    heads = []
    for a in range(H):
        s = (q[:, a] @ k[:, a].T * mx["scale"]).masked_fill(~past, -math.inf)
        heads.append(torch.softmax(s, -1) @ v[:, a] * gate[:, a:a + 1])
    return torch.cat(heads, -1) @ W[p + "o"].T


def poly_norm(z, coef, eps):
    return coef[0] * rms_unit(z, eps) + coef[1] * rms_unit(z ** 2, eps) + coef[2] * rms_unit(z ** 3, eps) + coef[3]


def feed_forward_dense(h, W, p, eps):
    return poly_norm(h @ W[p + "up"].T, W[p + "act"], eps) @ W[p + "down"].T


def clamped_expert(x, W, p, limit):
    g = torch.clamp(x @ W[p + "gate"].T, max=limit)
    u = torch.clamp(x @ W[p + "up"].T, -limit, limit)
    return (g * torch.sigmoid(1.702 * g) * (u + 1.0)) @ W[p + "down"].T


def route(h, W, p, ml):
    """-> chosen [T, top], weight [T, top] (the scores themselves)."""
    s = torch.sigmoid(h @ W[p + "router"].T)
    weight, chosen = torch.topk(s, ml["router"]["top"], dim=-1)
    return chosen, weight


def feed_forward_moe(h, W, p, ml):
    chosen, weight = route(h, W, p, ml)
    y = torch.zeros_like(h)
    for e in sorted(set(chosen.reshape(-1).tolist())):
        t, k = torch.nonzero(chosen == e, as_tuple=True)
        y.index_add_(0, t, clamped_expert(weight[t, k].unsqueeze(-1) * h[t], W, f"{p}e{e}.", ml["expert"]["limit"]))  # the INPUT is weighted
    return y


def forward(config, W, tokens, residuals=None):
    """logits [T, vocab] of one sequence; residuals (a list) receives the stream after every layer."""
    eps, alpha = config["norm"]["eps"], config["postln_alpha"]
    x = W["embed"][torch.as_tensor(tokens, dtype=torch.long)] + position_vector(len(tokens), config["width"])
    cached = {}
    for i, layer in enumerate(config["layers"]):
        p, mx, ml = f"l{i}.", layer["mixer"], layer["mlp"]
        h = with_conv(x, W[p + "canon1"])
        if layer["type"] == "mingru":
            y = mixer_mingru(h, W, p + "mix.")
        else:
            if "kv_from" in mx:
                c = cached[mx["kv_from"]]
            else:
                c = cached[i] = latent_rows(h, W, p + "mix.", eps)
            y = mixer_latent(h, W, p + "mix.", mx, eps, c)
        x = norm_around_zero(alpha * x + y, W[p + "norm1"], eps)
        if ml is not None:
            h = with_conv(x, W[p + "canon2"])
            y = feed_forward_dense(h, W, p + "mlp.", eps) if ml["kind"] == "dense" else feed_forward_moe(h, W, p + "mlp.", ml)
            x = norm_around_zero(alpha * x + y, W[p + "norm2"], eps)
        if residuals is not None:
            residuals.append(x)
    return norm_around_zero(x, W["final.norm"], eps) @ W["head"].T


def greedy(config, W, prompt, n):
    ids = list(prompt)
    for _ in range(n):
        ids.append(int(torch.argmax(forward(config, W, ids)[-1])))
    return ids[len(prompt):]


# ------------------------------------------------------------------ small random models
def mingru(width=20, mlp=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def latent(heads=3, dim=12, vdim=10, kv_rank=16, q_rank=14, scale=None, kv_from=None, mlp=None):
    mx = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": kv_rank, "q_rank": q_rank, "scale": scale if scale is not None else dim ** -0.5}
    if kv_from is not None:
        mx["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": mx, "mlp": mlp}


def dense(ff=44):
    return {"kind": "dense", "ff": ff}


def moe(experts=5, top=2, ff=12, limit=0.9):
    return {"kind": "moe", "router": {"experts": experts, "top": top}, "expert": {"ff": ff, "limit": limit}}


def make_config(layers, width=36, vocab=50, eps=1e-5, alpha=1.7, taps=3):
    return {"architecture": "Zasapel", "width": width, "vocab": vocab, "canon": {"taps": taps}, "norm": {"eps": eps}, "postln_alpha": alpha,
            "layers": layers}


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
        put(p + "norm1", d, std=0.2)
        put(p + "canon1", d, config["canon"]["taps"], std=0.4)
        if layer["type"] == "mingru":
            n = mx["width"]
            for k in ("z", "x", "g"):
                put(p + "mix." + k, n, d)
            put(p + "mix.z.b", n, std=0.5, mean=-1.0)
            put(p + "mix.x.b", n, std=0.5)
            put(p + "mix.o", d, n, std=2.0 / math.sqrt(n))
        elif layer["type"] == "latent_attention":
            H, r, rq = mx["heads"], mx["kv_rank"], mx["q_rank"]
            put(p + "mix.dq", rq, d)
            put(p + "mix.dq.norm", rq, std=0.2, mean=1.0)
            put(p + "mix.uq", H * mx["dim"], rq, std=2.0 / math.sqrt(rq))
            if "kv_from" not in mx:
                put(p + "mix.dkv", r, d)
                put(p + "mix.dkv.norm", r, std=0.2, mean=1.0)
            put(p + "mix.uk", H * mx["dim"], r)
            put(p + "mix.uv", H * mx["vdim"], r)
            put(p + "mix.g", H, d)
            put(p + "mix.o", d, H * mx["vdim"], std=2.0 / math.sqrt(H * mx["vdim"]))
        if ml is None:
            continue
        put(p + "norm2", d, std=0.2)
        put(p + "canon2", d, config["canon"]["taps"], std=0.4)
        if ml["kind"] == "dense":
            put(p + "mlp.up", ml["ff"], d)
            put(p + "mlp.act", 4, std=0.6, mean=0.3)
            put(p + "mlp.down", d, ml["ff"])
        elif ml["kind"] == "moe":
            for e in range(ml["router"]["experts"]):
                put(f"{p}mlp.e{e}.gate", ml["expert"]["ff"], d, std=1.5 / math.sqrt(d))
                put(f"{p}mlp.e{e}.up", ml["expert"]["ff"], d, std=1.5 / math.sqrt(d))
                put(f"{p}mlp.e{e}.down", d, ml["expert"]["ff"])
            put(p + "mlp.router", ml["router"]["experts"], d)
    put("final.norm", d, std=0.2)
    put("head", V, d)
    return {k: v.double() for k, v in W.items()}, W


def rel_err(got, want):
    got, want = np.asarray(got, np.float64), np.asarray(want, np.float64)
    return float(np.linalg.norm(got - want) / max(np.linalg.norm(want), 1e-30))
