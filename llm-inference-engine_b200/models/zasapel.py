"""Zasapel: a decoder-only design whose norm takes the sum, x <- rms(alpha * x + sublayer(x')) * (1 + w), and whose sublayers read
x' = x + conv(x), a short causal convolution over time on every channel (its last inputs are part of a sequence's state).  A sinusoidal
position vector joins the embedding; nothing else carries positions.  Two token mixers --

  * "mingru": a gated recurrence whose gates read the current token only, s <- (1 - z) s + z c with z = sigmoid(W_z h + b) and
    c = u + 1/2 (u >= 0) or sigmoid(u), u = W_x h + b; one fp32 state vector; output W_o (s * silu(W_g h));
  * "latent_attention": keys and values of all heads are up-projections of one cached RMS-normed row per position, queries come through a
    normed low-rank row of their own, plain causal softmax, ONE sigmoid gate per head; a layer with "kv_from": j reads layer j's rows
    through its own up-projections --

beside a dense feed-forward W_down act(W_up h), act = a n(z) + b n(z^2) + c n(z^3) + e with n(v) = v / rms(v), or routed experts (sigmoid
router, the chosen scores weigh the experts' INPUTS and are not renormalised, clamped gated experts).  The final norm has the layers' form.

config.json gives every size and constant; this module turns it plus the checkpoint's tensors into the layer list of hybrid.HybridDecoder:
projections that read the same input are fused into one matrix (z | x | gate; dq | dkv | gate), W_uk is stored per head transposed,
an expert's gate and up rows are stacked, the experts' matrices are stacked, norm weights become 1 + w in fp32, the convolutions' taps
come first in their layout."""
import importlib
import os

from . import register

POSITION_BASE = 10000.0   # sinusoidal position vector
GATE_SLOPE = 1.702        # of the experts' gate g * sigmoid(slope * g)


def _pkg(sub=None):
    base = __package__.rsplit(".", 1)[0]
    return importlib.import_module(base + ("." + sub if sub else ""))


def layer_specs(config):
    """The integer / float side of every layer, straight from config.json (no tensors yet)."""
    m = _pkg()
    taps = int((config.get("canon") or {}).get("taps") or 0)   # absent: the sublayers read x itself
    out = []
    for i, layer in enumerate(config["layers"]):
        mx, kind = layer["mixer"], layer["type"]
        if kind == "mingru":
            spec = dict(mixer=m.MIXER_MINGRU, heads=1, kv_heads=1, dim=1, vdim=int(mx["width"]))
        elif kind == "latent_attention":
            kv_from = mx.get("kv_from")
            spec = dict(mixer=m.MIXER_LATENT, heads=int(mx["heads"]), kv_heads=1, dim=int(mx["dim"]), vdim=int(mx["vdim"]), kv_rank=int(mx["kv_rank"]),
                        q_rank=int(mx["q_rank"]), scale=float(mx["scale"]), head_gate=1, kv_from=-1 if kv_from is None else int(kv_from))
            if spec["kv_from"] >= i:
                raise ValueError(f"layer {i}: kv_from {spec['kv_from']} is not an earlier layer")
        else:
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        spec.update(norm=m.NORM_RMS_SUM, in_taps=taps)
        mlp = layer.get("mlp")
        if mlp is None:
            spec.update(mlp=m.MLP_NONE)
        elif mlp.get("kind") == "dense":
            spec.update(mlp=m.MLP_DENSE, expert_ff=int(mlp["ff"]), act=m.ACT_POLYNORM, gated=0)
        elif mlp.get("kind") == "moe":
            spec.update(mlp=m.MLP_MOE, route=m.ROUTE_SIGMOID, experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]),
                        expert_ff=int(mlp["expert"]["ff"]), act=m.ACT_CLAMP_GLU, act_limit=float(mlp["expert"].get("limit") or 0.0), act_slope=GATE_SLOPE,
                        gated=1)
        else:
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        out.append(spec)
    return out


def norm_weight(get, name, device):
    """A norm weight stored as its distance from one."""
    import torch

    return (1.0 + get(name).float()).reshape(-1).to(device=device, dtype=torch.float32).contiguous()


def fuse_layer(spec, get, dtype, device):
    """Adds the device tensors of one layer to its spec.  get(name) -> CPU tensor of the checkpoint ('mix.z', 'mlp.e0.up', ...)."""
    import torch

    m = _pkg()

    def mat(*names):
        ts = [get(n) for n in names]
        return (torch.cat(ts, 0) if len(ts) > 1 else ts[0]).to(device=device, dtype=dtype).contiguous()

    def vec(*names):
        return torch.cat([get(n).float().reshape(-1) for n in names]).to(device=device, dtype=torch.float32).contiguous()

    def conv(name):
        return get(name).float().t().to(device).contiguous()   # [taps, width]

    spec.update(w_out=mat("mix.o"), norm1=norm_weight(get, "norm1", device))
    if spec["in_taps"]:
        spec["in_conv1"] = conv("canon1")
    if spec["mixer"] == m.MIXER_MINGRU:
        spec.update(w_in=mat("mix.z", "mix.x", "mix.g"), b_in=vec("mix.z.b", "mix.x.b"))
    else:
        H, dim, vdim, rank = spec["heads"], spec["dim"], spec["vdim"], spec["kv_rank"]
        own = spec["kv_from"] < 0
        spec.update(w_in=mat("mix.dq", "mix.dkv", "mix.g") if own else mat("mix.dq", "mix.g"), dq_norm=vec("mix.dq.norm"), w_uq=mat("mix.uq"),
                    w_uk_t=get("mix.uk").reshape(H, dim, rank).transpose(1, 2).to(device=device, dtype=dtype).contiguous(),
                    w_uv=get("mix.uv").reshape(H, vdim, rank).to(device=device, dtype=dtype).contiguous())
        if own:
            spec["kv_norm"] = vec("mix.dkv.norm")
    if spec["mlp"] == m.MLP_NONE:
        return spec
    spec["norm2"] = norm_weight(get, "norm2", device)
    if spec["in_taps"]:
        spec["in_conv2"] = conv("canon2")
    if spec["mlp"] == m.MLP_DENSE:
        spec.update(w_up=mat("mlp.up"), w_down=mat("mlp.down"), act_coef=vec("mlp.act"))
    else:
        E = spec["experts"]
        spec.update(w_router=mat("mlp.router"),
                    w_up=torch.stack([torch.cat([get(f"mlp.e{e}.gate"), get(f"mlp.e{e}.up")], 0) for e in range(E)]).to(device=device, dtype=dtype).contiguous(),
                    w_down=torch.stack([get(f"mlp.e{e}.down") for e in range(E)]).to(device=device, dtype=dtype).contiguous())
    return spec


@register("Zasapel")
class ZasapelModel:
    """config + tensors -> a HybridDecoder.  `tensors`: name -> CPU tensor with the checkpoint's names ('embed', 'l0.mix.z', ..., 'head')."""

    def __init__(self, config, tensors, dtype="bfloat16", device="cuda:0", max_tokens=2048, max_seqs=4, max_pages_per_seq=None):
        import torch

        m = _pkg()
        tdt = {"bfloat16": torch.bfloat16, "float16": torch.float16, "float32": torch.float32}[dtype] if isinstance(dtype, str) else dtype
        self.config, self.width, self.vocab = config, int(config["width"]), int(config["vocab"])
        self.eps = float(config["norm"]["eps"])
        specs = layer_specs(config)
        for i, spec in enumerate(specs):
            fuse_layer(spec, lambda n, i=i: tensors[f"l{i}.{n}"], tdt, device)
        if max_pages_per_seq is None:
            max_pages_per_seq = (max_tokens + m.KV_PAGE_SIZE - 1) // m.KV_PAGE_SIZE
        self.engine = _pkg("hybrid").HybridDecoder(
            self.width, self.vocab, self.eps, specs, tensors["embed"].to(device=device, dtype=tdt).contiguous(),
            norm_weight(lambda n: tensors[n], "final.norm", device), tensors["head"].to(device=device, dtype=tdt).contiguous(), tdt, device, max_tokens,
            max_seqs, max_pages_per_seq, final_norm_kind=m.NORM_RMS_SUM, pos_base=POSITION_BASE, residual_scale=float(config["postln_alpha"]))

    @classmethod
    def from_pretrained(cls, model_dir, config, dtype="bfloat16", device="cuda:0", **limits):
        tensors = _pkg("weights").read_safetensors(os.path.join(model_dir, "model.safetensors"))
        return cls(config, tensors, dtype=dtype, device=device, **limits)
