"""Pamulix: a decoder-only design whose layers norm a sublayer's OUTPUT only, x <- x + m * layernorm(sublayer(x)) (weight, no bias; one m for
the model), with two token mixers --

  * "latent_attention": keys and values of all heads are up-projections (W_uk, W_uv) of one cached RMS-normed row per position, plus one
    rotated key part shared by the heads; queries come through a normed low-rank row of their own, a head is [dim un-rotated | rot_dim
    rotated]; rotation in neighbouring pairs with YaRN-scaled frequencies; plain causal softmax, no gate, no sink;
  * "attention": grouped-query attention without rotation; per-head RMS norm of q and k (one weight each, shared by the heads); a linear
    distance bias per head, slope 2^(-8 (h + 1) / heads); a block-diagonal causal mask (blocks of mask.size positions from position 0);
    softmax with one added to the denominator; with "v_mix" the values are mixed with those of the first such layer, v <- (1 - lambda) v +
    lambda v_first, before they are cached --

and mixture-of-experts feed-forwards: router logits + bias, the `top` largest, softmax over the chosen ones as weights on the outputs of gated
silu experts.  The final norm has the layers' form.

config.json gives every size and constant; this module turns it plus the checkpoint's tensors into the layer list of hybrid.HybridDecoder:
projections that read the same input are fused into one matrix (q | k | v; dq | dkv), W_uk is stored per head transposed, an expert's gate and
up rows are stacked, the experts' matrices are stacked, slopes and frequencies become small tables."""
import importlib
import os

from . import register, rotation


def _pkg(sub=None):
    base = __package__.rsplit(".", 1)[0]
    return importlib.import_module(base + ("." + sub if sub else ""))


def rotation_table(rot):
    """rot of a latent layer -> (turns per position of every pair, amplitude)."""
    dims, base, scaling = int(rot["dims"]), float(rot["base"]), rot.get("scaling")
    if scaling:
        freq, amp = rotation.yarn(dims, base, *(float(scaling[k]) for k in ("factor", "original", "fast", "slow")))
    else:
        freq, amp = rotation.plain_frequencies(dims, base), 1.0
    return rotation.turns(freq), amp


def distance_slopes(heads):
    return [2.0 ** (-8.0 * (h + 1) / heads) for h in range(heads)]


def layer_specs(config):
    """The integer / float side of every layer, straight from config.json (no tensors yet)."""
    m = _pkg()
    out, first_values = [], None
    for i, layer in enumerate(config["layers"]):
        mx, kind = layer["mixer"], layer["type"]
        spec = dict(norm=m.NORM_LN_POST, heads=int(mx["heads"]), dim=int(mx["dim"]), vdim=int(mx.get("vdim", mx["dim"])), scale=float(mx["scale"]))
        if kind == "latent_attention":
            rot_dim = int(mx.get("rot_dim") or 0)
            spec.update(mixer=m.MIXER_LATENT, kv_heads=1, kv_rank=int(mx["kv_rank"]), q_rank=int(mx["q_rank"]), rot_dim=rot_dim, head_gate=2)
            if rot_dim:
                table, amp = rotation_table(mx["rot"])
                spec.update(rot_dims=2 * len(table), rot_base=float(mx["rot"]["base"]), rot_pairs=1, rot_amp=amp, turns=table)
        elif kind == "attention":
            mask = mx.get("mask") or {}
            spec.update(mixer=m.MIXER_ATTN_SCORED, attn_weight=m.ATTN_SOFTMAX, kv_heads=int(mx.get("kv_heads", mx["heads"])), chunk=int(mask.get("size") or 0))
            if mx.get("v_mix"):
                sizes = (spec["kv_heads"], spec["vdim"])
                if first_values is None:
                    first_values, spec["v_share"] = sizes, 1
                else:
                    if sizes != first_values:
                        raise ValueError(f"layer {i}: values of {sizes[0]} x {sizes[1]} cannot be mixed with the first layer's {first_values[0]} x {first_values[1]}")
                    spec["v_share"] = 2
        else:
            raise ValueError(f"layer {i}: unknown mixer type {kind!r}")
        mlp = layer.get("mlp")
        if mlp is None:
            spec.update(mlp=m.MLP_NONE)
        elif mlp.get("kind", "moe") == "moe":
            spec.update(mlp=m.MLP_MOE, route=m.ROUTE_SOFTMAX, experts=int(mlp["router"]["experts"]), top=int(mlp["router"]["top"]),
                        expert_ff=int(mlp["expert"]["ff"]), act=m.ACT_SILU, gated=1)
        else:
            raise ValueError(f"layer {i}: unknown feed-forward kind {mlp.get('kind')!r}")
        out.append(spec)
    return out


def fuse_layer(spec, get, dtype, device):
    """Adds the device tensors of one layer to its spec.  get(name) -> CPU tensor of the checkpoint ('mix.q', 'mlp.e0.up', ...)."""
    import torch

    m = _pkg()

    def mat(*names):
        ts = [get(n) for n in names]
        return (torch.cat(ts, 0) if len(ts) > 1 else ts[0]).to(device=device, dtype=dtype).contiguous()

    def vec(name):
        return get(name).to(device=device, dtype=torch.float32).reshape(-1).contiguous()

    H, dim, vdim = spec["heads"], spec["dim"], spec["vdim"]
    spec.update(w_out=mat("mix.o"), norm1=vec("norm1"))
    if spec["mixer"] == m.MIXER_LATENT:
        rank = spec["kv_rank"]
        spec.update(w_in=mat("mix.dq", "mix.dkv"), dq_norm=vec("mix.dq.norm"), w_uq=mat("mix.uq"), kv_norm=vec("mix.dkv.norm"),
                    w_uk_t=get("mix.uk").reshape(H, dim, rank).transpose(1, 2).to(device=device, dtype=dtype).contiguous(),
                    w_uv=get("mix.uv").reshape(H, vdim, rank).to(device=device, dtype=dtype).contiguous())
        if spec["rot_dim"]:
            spec["rot_turns"] = torch.tensor(spec["turns"], dtype=torch.float64, device=device)
    else:
        spec.update(w_in=mat("mix.q", "mix.k", "mix.v"), q_norm=vec("mix.q.norm"), k_norm=vec("mix.k.norm"),
                    dist_slope=torch.tensor(distance_slopes(H), dtype=torch.float32, device=device),
                    sink=torch.zeros(H, dtype=torch.float32, device=device))   # one added to the denominator: a sink whose logit is 0
        if spec.get("v_share") == 2:
            spec["v_lambda"] = float(get("mix.vmix").float().reshape(()))
    if spec["mlp"] == m.MLP_NONE:
        return spec
    E = spec["experts"]
    spec.update(norm2=vec("norm2"), w_router=mat("mlp.router"), logit_bias=vec("mlp.router.b"),
                w_up=torch.stack([torch.cat([get(f"mlp.e{e}.gate"), get(f"mlp.e{e}.up")], 0) for e in range(E)]).to(device=device, dtype=dtype).contiguous(),
                w_down=torch.stack([get(f"mlp.e{e}.down") for e in range(E)]).to(device=device, dtype=dtype).contiguous())
    return spec


@register("Pamulix")
class PamulixModel:
    """config + tensors -> a HybridDecoder.  `tensors`: name -> CPU tensor with the checkpoint's names ('embed', 'l0.mix.q', ..., 'head')."""

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
            tensors["final.norm"].to(device=device, dtype=torch.float32).contiguous(), tensors["head"].to(device=device, dtype=tdt).contiguous(), tdt, device,
            max_tokens, max_seqs, max_pages_per_seq, final_norm_kind=m.NORM_LN_POST, branch_scale=float(config["residual_mult"]))

    @classmethod
    def from_pretrained(cls, model_dir, config, dtype="bfloat16", device="cuda:0", **limits):
        tensors = _pkg("weights").read_safetensors(os.path.join(model_dir, "model.safetensors"))
        return cls(config, tensors, dtype=dtype, device=device, **limits)
