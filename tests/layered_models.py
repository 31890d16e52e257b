"""Small seeded model directories for the tests of the layer-list decoders."""
import json
import os

import layered_oracle as O
import torch


def attention(heads=6, kv_heads=2, dim=40, scale=0.2, size=37, keep=3, ff=None, limit=1.1):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": dim, "scale": scale,
                                           "mask": {"size": size, "keep_first": keep}}, "mlp": mlp(ff, limit)}


def mlstm(heads=3, dim=24, vdim=40, cap=9.0, ff=None, limit=0.7):
    return {"type": "mlstm", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}, "mlp": mlp(ff, limit)}


def mlp(ff, limit):
    return None if ff is None else {"kind": "dense", "ff": ff, "limit": limit}


def config(layers, width=152, vocab=331, eps=1e-5):
    return {"architecture": "Keripel", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}


# every branch in one model: both mixers with and without a feed-forward, group sizes 3 and 1, odd sizes
def mixed_config():
    return config([attention(ff=200), mlstm(), attention(heads=4, kv_heads=4, dim=72, scale=0.11, size=100, keep=0),
                   mlstm(heads=1, dim=100, vdim=136, cap=4.0, ff=90)])


# ---- Kekevik ----------------------------------------------------------------------------------------------------------------------
def relu2(ff):
    return None if ff is None else {"kind": "dense", "ff": ff}


def decays(heads):
    """From a few tokens to a few hundred."""
    return [1.0 - 0.4 * 0.3 ** (4.5 * h / max(1, heads - 1)) for h in range(heads)]


def retention(heads=3, dim=24, vdim=40, base=5000.0, dims=None, decay=None, ff=None):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or decays(heads),
                                           "rot": {"base": base, "dims": dim if dims is None else dims}}, "mlp": relu2(ff)}


def lightning(heads=5, dim=20, vdim=36, decay=None, ff=None):
    return {"type": "lightning", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": decay or decays(heads)}, "mlp": relu2(ff)}


def capped(heads=6, kv_heads=2, dim=40, vdim=24, scale=0.3, cap=6.0, coef=0.7, every=19):
    return {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "softcap": cap, "q_temp": {"coef": coef, "every": every}}


def ssd(heads=6, vdim=20, state=28, groups=2, parts=3, conv=4):
    return {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": parts, "conv": conv}


def parallel(left=None, right=None, scales=(0.7, 1.3), ff=None):
    return {"type": "parallel", "mixer": {"left": left or capped(), "right": right or ssd(), "left_scale": scales[0], "right_scale": scales[1]}, "mlp": relu2(ff)}


def kekevik(layers, width=152, vocab=331, eps=1e-5, scale=3.5):
    return {"architecture": "Kekevik", "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width, "embedding": {"scale": scale}}


# every branch in one model: the three mixers with and without a feed-forward, shared and own queries and keys, odd sizes
def kekevik_mixed():
    return kekevik([parallel(ff=200), retention(), lightning(ff=90), parallel(capped(4, 4, 32, 72, 0.2, 20.0, -0.1, 7), ssd(4, 33, 70, 1, 2, 3)),
                    retention(2, 50, 66, 100.0, 30, ff=70), lightning(1, 70, 130)])


# ---- Kutepel ----------------------------------------------------------------------------------------------------------------------
STRETCH = {"factor": 5.0, "low": 1.5, "high": 6.0, "original": 90}


def experts(ff=40, n=12, top=3, groups=3, keep=2, scale=1.7):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": n, "groups": {"count": groups, "keep": keep}, "scale": scale, "top": top}}


def rotation(dims, base, scaling):
    return {"base": base, "dims": dims, **({} if scaling is None else {"scaling": scaling})}


def rotary(heads=6, kv_heads=2, dim=40, vdim=24, scale=0.25, dims=None, base=2000.0, scaling=None, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "rot": rotation(dim if dims is None else dims, base, scaling)}
    return {"type": "attention", "mixer": m if kv_from is None else {**m, "kv_from": kv_from}, "mlp": mlp}


def latent(heads=3, dim=20, rot_dim=12, vdim=28, rank=72, scale=0.3, base=700.0, scaling=None, mlp=None):
    return {"type": "latent_attention", "mixer": {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale,
                                                  "rot": rotation(rot_dim, base, scaling)}, "mlp": mlp}


def kutepel(layers, width=152, vocab=331, eps=1e-5, mult=0.4):
    return {"architecture": "Kutepel", "layers": layers, "norm": {"eps": eps}, "residual_mult": mult, "vocab": vocab, "width": width}


# every branch in one model: both mixers with and without experts, own and shared keys, with and without stretched frequencies
def kutepel_mixed():
    return kutepel([latent(mlp=experts()), rotary(scaling=STRETCH, mlp=experts(33, 10, 2, 5, 3, 0.8)), latent(5, 33, 30, 70, 130, 0.15, 1e4, STRETCH),
                    rotary(kv_from=1, scaling=STRETCH, mlp=experts(24, 7, 1, 1, 1, 1.0)), rotary(4, 4, 32, 72, 0.2, 20), rotary(12, 2, kv_from=1, dims=10, mlp=experts()),
                    latent(17, 16, 2, 8, 16, 0.3, 50.0, mlp=experts(64, 20, 4, 10, 2, 2.0))])


# ---- Naforax ----------------------------------------------------------------------------------------------------------------------
def gelu(ff=70):
    return {"kind": "dense", "ff": ff}


def moe(ff=40, n=11, top=3, limit=0.9, shared=(56, 1.3)):
    m = {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": n, "top": top}}
    return m if shared is None else {**m, "shared": {"ff": shared[0], "limit": shared[1]}}


def differential(heads=6, kv_heads=2, dim=20, vdim=28, scale=0.3, size=70, dims=12, base=900.0, diff=0.4, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size},
                                           "rot": {"base": base, "dims": dims}, "diff": diff}, "mlp": mlp}


def mingru(width=100, mlp=None):
    return {"type": "mingru", "mixer": {"width": width}, "mlp": mlp}


def mamba1(inner=90, state=12, rank=9, conv=4, mlp=None):
    return {"type": "mamba1", "mixer": {"inner": inner, "state": state, "dt_rank": rank, "conv": conv}, "mlp": mlp}


def naforax(layers, loop=(0, 1, 1), width=152, vocab=331, eps=1e-5, groups=4, taps=3, mult=0.6, cap=9.0):
    return {"architecture": "Naforax", "layers": layers, "loop": dict(zip(("start", "stop", "times"), loop)), "norm": {"eps": eps, "groups": groups},
            "canon": {"taps": taps}, "residual_mult": mult, "logit_softcap": cap, "vocab": vocab, "width": width}


# every branch in one model: all mixers inside and outside the loop, dense blocks, experts with and without a shared one, no block
def naforax_mixed():
    return naforax([mingru(mlp=moe()), differential(mlp=gelu()), mamba1(mlp=moe(24, 5, 1, 2.0, None)), differential(4, 4, 33, 40, 0.2, 100, 6, 50.0, 0.1, mlp=moe(33, 7, 7, 0.5)),
                    mamba1(77, 20, 3, 2), mingru(64, mlp=gelu(45)), differential(8, 1, 16, 72, 0.4, 37, 16, 2e4, 0.7)], loop=(1, 4, 3))


def write(path, cfg, weights):
    from oxibonsai_b200.convert import write_safetensors
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    write_safetensors(os.path.join(path, "model.safetensors"), {k: v.bfloat16() for k, v in weights.items()})
    return str(path)


class Model:
    """A model directory with its oracle weights."""

    def __init__(self, path, cfg, seed=0, tweak=None, scale=1.0):
        self.cfg = cfg
        w = O.random_weights(cfg, seed, scale)
        if tweak is not None:
            tweak(w)
            w = {k: v.bfloat16().float() for k, v in w.items()}
        self.path = write(path, cfg, w)
        self.w = {k: v.double() for k, v in w.items()}

    def tokens(self, n, seed=1):
        return torch.randint(0, self.cfg["vocab"], (n,), generator=torch.Generator().manual_seed(seed)).tolist()

    def logits(self, tokens):
        return O.forward(self.cfg, self.w, tokens)

    def greedy(self, prompt, n):
        """Greedy continuation and the smallest gap between the two best logits on the way."""
        seq, gap = list(prompt), float("inf")
        for _ in range(n):
            top = torch.topk(self.logits(seq)[-1], 2).values
            gap = min(gap, float(top[0] - top[1]))
            seq.append(int(self.logits(seq)[-1].argmax()))
        return seq[len(prompt):], gap
