#!/usr/bin/env python
"""Layer-list decoders beside the closest existing model: Keripel beside the generic-format Qwen3 engine with f16 weights,
Kekevik beside Keripel, Kutepel and Naforax beside Kekevik.

    python benchmarks/layered.py kernels [--width 4096] [--only ..]     the kernels and their counterparts, with roofline fractions
    python benchmarks/layered.py models --design kutepel [--sizes s,m]  prefill and decode throughput at equal parameter count

Random weights, random tokens.  Kernels: CUDA events around a CUDA graph of repeated launches that walks through enough copies
of its inputs to exceed L2; the roofline is the slower of bytes / measured copy bandwidth and FLOPs / measured bf16 GEMM rate.
"""
from __future__ import annotations

import argparse
import json
import os
import sys
import tempfile

sys.path.insert(0, os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
sys.path.insert(0, os.path.dirname(os.path.abspath(__file__)))

import torch

from kernels import peaks, time_us

F16 = 1


def keripel(width: int, repeats: int, vocab: int = 32000, window: int = 1024) -> dict:
    """``repeats`` times three recurrent layers and one attention layer with a feed-forward block."""
    m = {"type": "mlstm", "mixer": {"heads": max(2, width // 512), "dim": 256, "vdim": 512, "gate_cap": 15.0}, "mlp": None}
    a = {"type": "attention", "mixer": {"heads": width // 128, "kv_heads": max(1, width // 512), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
                                        "mask": {"size": window, "keep_first": 4}},
         "mlp": {"kind": "dense", "ff": 3 * width, "limit": 7.0}}
    return {"architecture": "Keripel", "layers": [m, m, m, a] * repeats, "norm": {"eps": 1e-6}, "vocab": vocab, "width": width}


def kekevik(width: int, repeats: int, vocab: int = 32000) -> dict:
    """``repeats`` times a lightning layer, two layers of attention beside a state-space mixer, and a retention layer."""
    H = width // 128
    decay = lambda n: [1.0 - 2.0 ** (-5.0 - 6.0 * i / max(1, n - 1)) for i in range(n)]
    ff = {"kind": "dense", "ff": 4 * width}
    light = {"type": "lightning", "mixer": {"heads": H, "dim": 128, "vdim": 128, "decay": decay(H)}, "mlp": ff}
    both = {"type": "parallel", "mlp": ff, "mixer": {
        "left": {"heads": H, "kv_heads": max(1, H // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5, "softcap": 50.0, "q_temp": {"coef": 0.1, "every": 4096}},
        "right": {"heads": width // 64, "vdim": 64, "state": 128, "groups": max(1, H // 4), "norm_groups": max(1, H // 4), "conv": 4},
        "left_scale": 0.5, "right_scale": 0.5}}
    n = max(1, width // 256)
    ret = {"type": "retention", "mlp": ff, "mixer": {"heads": n, "dim": 256, "vdim": 256, "decay": decay(n), "rot": {"base": 10000.0, "dims": 256}}}
    return {"architecture": "Kekevik", "layers": [light, both, both, ret] * repeats, "norm": {"eps": 1e-6}, "vocab": vocab, "width": width,
            "embedding": {"scale": float(width ** 0.5)}}


def kutepel(width: int, repeats: int, vocab: int = 32000, n: int = 32, top: int = 4) -> dict:
    """``repeats`` times two layers of latent attention, one of rotary attention with sinks and one on its keys and values, all with
    ``n`` experts of a quarter of the width."""
    H = width // 128
    moe = {"kind": "moe", "expert": {"ff": width // 4}, "router": {"experts": n, "groups": {"count": 8, "keep": 4}, "scale": 2.5, "top": top}}
    lat = {"type": "latent_attention", "mlp": moe, "mixer": {"heads": H, "dim": 128, "rot_dim": 64, "vdim": 128, "kv_rank": 512, "scale": 192 ** -0.5,
                                                             "rot": {"base": 10000.0, "dims": 64}}}
    m = {"heads": H, "kv_heads": max(1, H // 4), "dim": 128, "vdim": 128, "scale": 128 ** -0.5,
         "rot": {"base": 500000.0, "dims": 128, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 8192}}}
    layers = []
    for r in range(repeats):
        layers += [lat, lat, {"type": "attention", "mlp": moe, "mixer": m}, {"type": "attention", "mlp": moe, "mixer": {**m, "kv_from": 4 * r + 2}}]
    return {"architecture": "Kutepel", "layers": layers, "norm": {"eps": 1e-6}, "residual_mult": 0.5, "vocab": vocab, "width": width}


def naforax(width: int, repeats: int, vocab: int = 32000, n: int = 32, top: int = 4, times: int = 2) -> dict:
    """``repeats`` times a layer of differential attention with a dense block, a minGRU, a selective scan, and attention again, those with
    ``n`` experts of a quarter of the width and a shared one; the recurrent layers of the first repeat run ``times`` times."""
    H = width // 128
    moe = {"kind": "moe", "expert": {"ff": width // 4, "limit": 7.0}, "router": {"experts": n, "top": top}, "shared": {"ff": width // 2, "limit": 7.0}}
    a = {"heads": H, "kv_heads": max(1, H // 4), "dim": 64, "vdim": 128, "scale": 64 ** -0.5, "mask": {"size": 8192}, "rot": {"base": 500000.0, "dims": 64}, "diff": 0.5}
    layers = [{"type": "attention", "mlp": {"kind": "dense", "ff": 3 * width}, "mixer": a}, {"type": "mingru", "mlp": moe, "mixer": {"width": width}},
              {"type": "mamba1", "mlp": moe, "mixer": {"inner": 2 * width, "state": 16, "dt_rank": width // 16, "conv": 4}}, {"type": "attention", "mlp": moe, "mixer": a}]
    return {"architecture": "Naforax", "layers": layers * repeats, "loop": {"start": 1, "stop": 3, "times": times}, "norm": {"eps": 1e-6, "groups": 4},
            "canon": {"taps": 4}, "residual_mult": 0.5, "logit_softcap": 30.0, "vocab": vocab, "width": width}


def write_design(path: str, cfg: dict) -> int:
    """A model directory with random bf16 weights; returns the parameter count."""
    from oxibonsai_b200.convert import write_safetensors
    from oxibonsai_b200.models.registry import ARCHITECTURES
    config = ARCHITECTURES[cfg["architecture"]](cfg, "")
    os.makedirs(path, exist_ok=True)
    with open(os.path.join(path, "config.json"), "w") as f:
        json.dump(cfg, f)
    g = torch.Generator(device="cuda").manual_seed(0)
    t = {}
    for n, s in config.tensor_shapes().items():
        x = torch.randn(s, generator=g, device="cuda")
        x = 1 + 0.1 * x if "norm" in n else (0.3 * x if len(s) == 1 else x * s[-1] ** -0.5)
        t[n] = x.bfloat16().cpu()
    write_safetensors(os.path.join(path, "model.safetensors"), t)
    return config.param_count()


class Report:
    def __init__(self):
        p = peaks()
        self.hbm, self.flops = p.get("hbm_gbs", 6650.0), p.get("bf16_tflops", 1590.0)
        self.rows: list[dict] = []

    def add(self, kernel: str, case: str, us: float, nbytes: float, flops: float = 0.0, like: str = "") -> float:
        roof = max(nbytes / (self.hbm * 1e3), flops / (self.flops * 1e6))
        r = {"kernel": kernel, "case": case, "us": round(us, 2), "roofline_us": round(roof, 2), "frac": round(roof / us, 4), "like": like}
        self.rows.append(r)
        print(json.dumps(r), flush=True)
        return roof / us


def bench_linear(rep: Report, width: int, iters: int, profile: bool) -> None:
    from oxibonsai_b200.ops import cuda_ops as K
    from oxibonsai_b200.ops import layered_ops as L
    dev = torch.device("cuda")
    scratch = L.GemmScratch(dev, torch.zeros(1, dtype=torch.int32, device=dev))
    for name, n, k in (("proj", 3 * width + 16, width), ("gate_up", 6 * width, width), ("down", width, 3 * width)):
        copies = max(2, int(400e6 / (2 * n * k)) + 1)
        ws = []
        for i in range(copies):
            w = L.DenseWeight([torch.zeros(8, k, dtype=torch.bfloat16)], dev)
            w.n, w.data = n, torch.randn(n, k, device=dev).bfloat16()
            ws.append(w)
        for T in (1, 8, 32, 64, 256, 4096):
            x = torch.randn(T, k, device=dev).bfloat16()
            if name == "gate_up":                # an ungated block's up projection of the same bytes
                sq, turn = torch.empty(T, n, dtype=torch.bfloat16, device=dev), [0]

                def relu2():
                    turn[0] += 1
                    L.linear(ws[turn[0] % copies], x, T, sq, scratch, L.SQUARED_RELU)
                rep.add("linear, squared relu", f"up {n}x{k} T={T}", time_us(relu2, iters, profile), 2 * n * k + 2 * T * k + 2 * T * n, 2.0 * T * n * k)
            glu = L.Glu(7.0, 1.702, 1.0) if name == "gate_up" else None
            out = torch.empty(T, n // 2 if glu else n, dtype=torch.bfloat16 if glu else torch.float32, device=dev)
            it = [0]

            def ours():
                it[0] += 1
                L.linear(ws[it[0] % copies], x, T, out, scratch, glu)
            nbytes, flops = 2 * n * k + 2 * T * k + out.numel() * out.element_size(), 2.0 * T * n * k
            rep.add("linear", f"{name} {n}x{k} T={T}", time_us(ours, iters, profile), nbytes, flops)
            xf, xh = x.float(), x.half()
            of = torch.empty(T, n, device=dev)

            def like():                      # same bytes read as f16
                it[0] += 1
                w = ws[it[0] % copies].data
                if T == 1:
                    K.quant_gemv(F16, w.view(torch.uint8).view(-1), n, k, xf.view(-1), out=of.view(-1))
                elif T <= 32:
                    K.quant_gemv_batched(F16, w.view(torch.uint8).view(-1), n, k, xf, out=of)
                else:
                    K.dense_gemm_f16(w.view(torch.float16), xh, out=of, status=scratch.status)
            rep.add("quant_gemv" if T <= 32 else "dense_gemm_f16", f"{name} {n}x{k} T={T}", time_us(like, iters, profile), 2 * n * k + 2 * T * k + 4 * T * n,
                    flops, "linear")


def bench_attention(rep: Report, width: int, iters: int, profile: bool) -> None:
    from oxibonsai_b200.ops import cuda_ops as K
    from oxibonsai_b200.ops import layered_ops as L
    dev = torch.device("cuda")
    nq, nkv, hd, page = width // 128, max(1, width // 512), 128, 64
    i32 = dict(dtype=torch.int32, device=dev)
    for B, ctx in ((1, 4096), (8, 4096), (64, 1024)):
        npages = ctx // page
        copies = max(2, int(300e6 / (2 * B * ctx * nkv * hd)) + 1)
        pools = [torch.randn(B * npages, nkv, page, hd, device=dev).bfloat16() for _ in range(copies)]
        rk = torch.ones(B * npages, nkv, page, device=dev)
        bt = torch.arange(B * npages, **i32).view(B, npages)
        pos, slots = torch.full((B,), ctx - 1, **i32), torch.arange(B, **i32)
        ld = (nq + nkv) * hd + nq
        proj = torch.randn(B, ld, device=dev)
        w1, slopes = torch.ones(hd, device=dev), torch.full((nq,), 0.01, device=dev)
        out = torch.zeros(B, nq * hd, dtype=torch.bfloat16, device=dev)
        calls = [L.MixerCall([proj, w1, w1, slopes, pos, slots, bt, p, rk, None, out, *[None] * 5],
                             [ld, 0, nq * hd, 0, (nq + nkv) * hd, nq * hd, nq, nkv, hd, hd, npages, page, 0, 0, 1, 0, 0, 0, 1, 0], [1e-6, hd ** -0.5, 1.0, 0.0, 0.0, 1.0, 0.0, 1.0]) for p in pools]
        it = [0]
        split = 1
        while split < 8 and B * nkv * split * 2 <= 160:
            split *= 2

        def ours():
            it[0] += 1
            K.check(L.lib().bonsai_lay_attn_decode(*calls[it[0] % copies].args, B, split, K.stream()), "attn_decode")
        kv_row = 2 * B * ctx * nkv * hd
        rep.add("attn_decode", f"B={B} ctx={ctx} heads={nq}/{nkv}", time_us(ours, iters, profile), kv_row, 4.0 * B * ctx * nq * hd)
        vp = [p.view(torch.float16) for p in pools]
        q, o = torch.randn(B, nq, hd, device=dev), torch.empty(B, nq, hd, device=dev)

        def like():
            it[0] += 1
            K.attn_decode(q, pos, bt, nq, nkv, hd, K.KV_F16, page, vp[it[0] % copies], vp[(it[0] + 1) % copies], nsplit=16, out=o)
        rep.add("attn_decode (f16 K and V)", f"B={B} ctx={ctx} heads={nq}/{nkv}", time_us(like, iters, profile), 2 * kv_row, 4.0 * B * ctx * nq * hd, "attn_decode")
    T, npages = 4096, 64
    pool, rk = torch.randn(npages, nkv, page, hd, device=dev).bfloat16(), torch.ones(npages, nkv, page, device=dev)
    bt, pos, slots = torch.arange(npages, **i32).view(1, -1), torch.arange(T, **i32), torch.zeros(T, **i32)
    proj, out = torch.randn(T, ld, device=dev), torch.zeros(T, nq * hd, dtype=torch.bfloat16, device=dev)
    tpt = 64 // (nq // nkv)
    entries = torch.tensor([0, T, 0, 0], **i32)
    tiles = torch.tensor([[0, t] for t in range(0, T, tpt)], **i32)
    for window in (0, 1024):
        call = L.MixerCall([proj, w1, w1, slopes, pos, slots, bt, pool, rk, None, out, *[None] * 5],
                           [ld, 0, nq * hd, 0, (nq + nkv) * hd, nq * hd, nq, nkv, hd, hd, npages, page, window, 4, 1, 0, 0, 0, 1, 0], [1e-6, hd ** -0.5, 1.0, 0.0, 0.0, 1.0, 0.0, 1.0])

        def ours():
            K.check(L.lib().bonsai_lay_attn_prompt(*call.args, entries.data_ptr(), tiles.data_ptr(), len(tiles), K.stream()), "attn_prompt")
        pairs = T * (T + 1) / 2 if not window else T * window - window * (window - 1) / 2 + 4 * (T - window)
        rep.add("attn_prompt", f"T={T} window={window or 'all'} heads={nq}/{nkv}", time_us(ours, 10, profile), 4 * T * ld + 2 * T * nkv * hd + 2 * T * nq * hd,
                4.0 * pairs * nq * hd)

    def append():
        K.check(L.lib().bonsai_lay_attn_append(*call.args, 0, T, 0, K.stream()), "attn_append")
    rep.add("attn_append", f"T={T}", time_us(append, iters, profile), 6 * T * nkv * hd)
    q, o16 = torch.randn(T, nq, hd, device=dev), torch.empty(T, nq * hd, dtype=torch.float16, device=dev)
    kp, vp = torch.randn(npages, nkv, page, hd, device=dev).half(), torch.randn(npages, nkv, page, hd, device=dev).half()
    rep.add("attn_prefill", f"T={T} heads={nq}/{nkv}", time_us(lambda: K.attn_prefill(q, 0, bt[0], nq, nkv, hd, K.KV_F16, page, kp, vp, out=o16), 10, profile),
            4 * T * nq * hd + 4 * T * nkv * hd + 2 * T * nq * hd, 4.0 * T * (T + 1) / 2 * nq * hd, "attn_prompt")


def bench_capped_attention(rep: Report, width: int, iters: int, profile: bool) -> None:
    """Attention with separate values, capped scores and a query temperature; the like kernels are those of bench_attention."""
    from oxibonsai_b200.ops import cuda_ops as K
    from oxibonsai_b200.ops import layered_ops as L
    dev = torch.device("cuda")
    nq, nkv, hd, page = width // 128, max(1, width // 512), 128, 64
    i32 = dict(dtype=torch.int32, device=dev)
    ld = (nq + 2 * nkv) * hd

    def call(proj, pos, slots, bt, k, v, out, cap=50.0):
        return L.MixerCall([proj, None, None, None, pos, slots, bt, k, None, v, out, *[None] * 5],
                           [ld, 0, nq * hd, (nq + nkv) * hd, -1, nq * hd, nq, nkv, hd, hd, bt.shape[1], page, 0, 0, 1, 0, 0, 0, 1, 0], [1e-6, hd ** -0.5, 0.5, cap, 0.1, 4096.0, 0.0, 1.0])
    for B, ctx in ((1, 4096), (8, 4096), (64, 1024)):
        npages = ctx // page
        copies = max(2, int(300e6 / (4 * B * ctx * nkv * hd)) + 1)
        pools = [[torch.randn(B * npages, nkv, page, hd, device=dev).bfloat16() for _ in range(2)] for _ in range(copies)]
        bt = torch.arange(B * npages, **i32).view(B, npages)
        pos, slots, proj = torch.full((B,), ctx - 1, **i32), torch.arange(B, **i32), torch.randn(B, ld, device=dev)
        out = torch.zeros(B, nq * hd, dtype=torch.bfloat16, device=dev)
        calls = [call(proj, pos, slots, bt, *p, out) for p in pools]
        it, split = [0], 1
        while split < 8 and B * nkv * split * 2 <= 160:
            split *= 2

        def ours():
            it[0] += 1
            K.check(L.lib().bonsai_lay_attn_decode(*calls[it[0] % copies].args, B, split, K.stream()), "attn_decode")
        rep.add("attn_decode, capped, K and V", f"B={B} ctx={ctx} heads={nq}/{nkv}", time_us(ours, iters, profile), 4 * B * ctx * nkv * hd, 4.0 * B * ctx * nq * hd)
    T, npages = 4096, 64
    k, v = (torch.randn(npages, nkv, page, hd, device=dev).bfloat16() for _ in range(2))
    bt, pos, slots = torch.arange(npages, **i32).view(1, -1), torch.arange(T, **i32), torch.zeros(T, **i32)
    proj, out = torch.randn(T, ld, device=dev), torch.zeros(T, nq * hd, dtype=torch.bfloat16, device=dev)
    entries = torch.tensor([0, T, 0, 0], **i32)
    tiles = torch.tensor([[0, t] for t in range(0, T, 64 // (nq // nkv))], **i32)
    for cap in (50.0, 0.0):
        c = call(proj, pos, slots, bt, k, v, out, cap)
        fn = lambda: K.check(L.lib().bonsai_lay_attn_prompt(*c.args, entries.data_ptr(), tiles.data_ptr(), len(tiles), K.stream()), "attn_prompt")
        rep.add("attn_prompt, K and V", f"T={T} heads={nq}/{nkv} cap={cap}", time_us(fn, 10, profile), 4 * T * ld + 4 * T * nkv * hd + 2 * T * nq * hd,
                4.0 * T * (T + 1) / 2 * nq * hd)
    fn = lambda: K.check(L.lib().bonsai_lay_attn_append(*c.args, 0, T, 0, K.stream()), "attn_append")
    rep.add("attn_append, K and V", f"T={T}", time_us(fn, iters, profile), 12 * T * nkv * hd)


def bench_rotary(rep: Report, width: int, iters: int, profile: bool) -> None:
    """Rotated heads with sinks; the like kernels are those of bench_capped_attention."""
    from oxibonsai_b200.ops import cuda_ops as K
    from oxibonsai_b200.ops import layered_ops as L
    dev = torch.device("cuda")
    nq, nkv, hd, page = width // 128, max(1, width // 512), 128, 64
    i32 = dict(dtype=torch.int32, device=dev)
    ld = (nq + 2 * nkv) * hd
    rot, sinks = torch.randn(4096, hd // 2, 2, device=dev), torch.ones(nq, device=dev)

    def call(proj, pos, slots, bt, k, v, out):
        return L.MixerCall([proj, None, None, None, pos, slots, bt, k, None, v, out, sinks, rot, None, None, None],
                           [ld, 0, nq * hd, (nq + nkv) * hd, -1, nq * hd, nq, nkv, hd, hd, bt.shape[1], page, 0, 0, 0, hd, 1, 0, 1, 0], [1e-6, hd ** -0.5, 1.0, 0.0, 0.0, 1.0, 0.0, 1.0])
    for B, ctx in ((1, 4096), (8, 4096), (64, 1024)):
        npages = ctx // page
        copies = max(2, int(300e6 / (4 * B * ctx * nkv * hd)) + 1)
        pools = [[torch.randn(B * npages, nkv, page, hd, device=dev).bfloat16() for _ in range(2)] for _ in range(copies)]
        bt = torch.arange(B * npages, **i32).view(B, npages)
        pos, slots, proj = torch.full((B,), ctx - 1, **i32), torch.arange(B, **i32), torch.randn(B, ld, device=dev)
        out = torch.zeros(B, nq * hd, dtype=torch.bfloat16, device=dev)
        calls = [call(proj, pos, slots, bt, *p, out) for p in pools]
        it, split = [0], 1
        while split < 8 and B * nkv * split * 2 <= 160:
            split *= 2

        def ours():
            it[0] += 1
            K.check(L.lib().bonsai_lay_attn_decode(*calls[it[0] % copies].args, B, split, K.stream()), "attn_decode")
        rep.add("attn_decode, rotated, sinks", f"B={B} ctx={ctx} heads={nq}/{nkv}", time_us(ours, iters, profile), 4 * B * ctx * nkv * hd, 4.0 * B * ctx * nq * hd)
    T, npages = 4096, 64
    k, v = (torch.randn(npages, nkv, page, hd, device=dev).bfloat16() for _ in range(2))
    bt, pos, slots = torch.arange(npages, **i32).view(1, -1), torch.arange(T, **i32), torch.zeros(T, **i32)
    proj, out = torch.randn(T, ld, device=dev), torch.zeros(T, nq * hd, dtype=torch.bfloat16, device=dev)
    entries = torch.tensor([0, T, 0, 0], **i32)
    tiles = torch.tensor([[0, t] for t in range(0, T, 64 // (nq // nkv))], **i32)
    c = call(proj, pos, slots, bt, k, v, out)
    fn = lambda: K.check(L.lib().bonsai_lay_attn_prompt(*c.args, entries.data_ptr(), tiles.data_ptr(), len(tiles), K.stream()), "attn_prompt")
    rep.add("attn_prompt, rotated, sinks", f"T={T} heads={nq}/{nkv}", time_us(fn, 10, profile), 4 * T * ld + 4 * T * nkv * hd + 2 * T * nq * hd, 4.0 * T * (T + 1) / 2 * nq * hd)
    fn = lambda: K.check(L.lib().bonsai_lay_attn_append(*c.args, 0, T, 0, K.stream()), "attn_append")
    rep.add("attn_append, rotated", f"T={T}", time_us(fn, iters, profile), 12 * T * nkv * hd)


def bench_latent(rep: Report, width: int, iters: int, profile: bool, splits: int = 0, cluster: int = 0, prompts: bool = True) -> None:
    """Latent attention; the like kernels are those of bench_capped_attention (and of bench_linear for the expansion)."""
    from oxibonsai_b200.models.layered import CONTEXT_TILE
    from oxibonsai_b200.ops import cuda_ops as K
    from oxibonsai_b200.ops import layered_ops as L
    dev, lib = torch.device("cuda"), L.lib()
    nq, dim, rot, vd, rank, page = width // 128, 128, 64, 128, 512, 64
    row, i32, bf16 = lib.bonsai_lay_latent_row(rank, rot), dict(dtype=torch.int32, device=dev), dict(dtype=torch.bfloat16, device=dev)
    q_w, g_w = nq * (dim + rot), nq * vd
    ld = q_w + rank + rot + g_w
    table, ones, sms = torch.randn(4096, rot // 2, 2, device=dev), torch.ones(rank, device=dev), torch.cuda.get_device_properties(dev).multi_processor_count

    def call(T, pos, slots, bt, pool, keys, values, parts):
        proj, out = torch.randn(T, ld, device=dev), torch.zeros(T, g_w, **bf16)
        n = min(T, 256)
        return L.MixerCall([proj, ones, table, pos, slots, bt, pool, keys, values, torch.randn(n, nq, row, device=dev).bfloat16() * 0.01,
                            torch.zeros(parts, nq, rank, device=dev), torch.ones(parts, nq, 2, device=dev), torch.zeros(1, **i32), out],
                           [ld, 0, q_w, q_w + rank, q_w + rank + rot, g_w, nq, dim, rot, vd, rank, bt.shape[1], page, n, parts, pool.shape[0]],
                           [1e-6, 192 ** -0.5, 1.0])
    for B, ctx in ((1, 4096), (8, 4096), (64, 1024)):
        npages = ctx // page
        copies = max(2, int(300e6 / (2 * B * ctx * row)) + 1)
        bt = torch.arange(B * npages, **i32).view(B, npages)
        pos, slots = torch.full((B,), ctx - 1, **i32), torch.arange(B, **i32)
        wcopies = int(300e6 / (2 * nq * rank * dim)) + 1
        ws = [[torch.randn(nq, rank, dim, device=dev).bfloat16() * 0.05, torch.randn(nq, vd, rank, device=dev).bfloat16() * 0.05] for _ in range(wcopies)]
        groups = -(-nq // lib.bonsai_lay_latent_group(nq))
        n = 1
        while 2 * n <= min(lib.bonsai_lay_latent_max_splits(), sms // (B * groups), -(-ctx // 64)):
            n *= 2
        n, cl = splits or n, min(splits or n, cluster or (lib.bonsai_lay_latent_max_cluster() if B * groups * n <= 64 else 4))
        calls = [call(B, pos, slots, bt, torch.randn(B * npages, page, row, device=dev).bfloat16(), *ws[i % wcopies], B * (n // cl)) for i in range(copies)]
        wcalls = [call(B, pos, slots, bt, torch.zeros(B * npages, page, row, **bf16), *w, B * (n // cl)) for w in ws]
        it = [0]

        def turn(fn, among):
            def run():
                it[0] += 1
                fn(among[it[0] % len(among)].args)
            return run
        query = turn(lambda a: K.check(lib.bonsai_lay_latent_query(*a, B, K.stream()), "latent_query"), wcalls)
        decode = turn(lambda a: K.check(lib.bonsai_lay_latent_decode(*a, B, n, cl, K.stream()), "latent_decode"), calls)
        value = turn(lambda a: K.check(lib.bonsai_lay_latent_value(*a, B, n // cl, K.stream()), "latent_value"), wcalls)
        case = f"B={B} ctx={ctx} heads={nq} {rank}+{rot} splits={n}/{cl}"
        rep.add("latent_query", case, time_us(query, iters, profile), 2 * nq * rank * dim + 4 * B * ld + 2 * B * nq * row, 2.0 * B * nq * rank * dim)
        rep.add("latent_decode", case, time_us(decode, iters, profile), 2 * B * ctx * row, 2.0 * B * ctx * nq * (2 * rank + rot))
        rep.add("latent_value", case, time_us(value, iters, profile), 2 * nq * rank * vd + 4 * B * (n // cl) * nq * rank, 2.0 * B * nq * rank * vd)

        def both():
            it[0] += 1
            a, w = calls[it[0] % copies].args, wcalls[it[0] % wcopies].args
            K.check(lib.bonsai_lay_latent_query(*w, B, K.stream()), "latent_query")
            K.check(lib.bonsai_lay_latent_decode(*a, B, n, cl, K.stream()), "latent_decode")
            K.check(lib.bonsai_lay_latent_value(*w, B, n // cl, K.stream()), "latent_value")
        rep.add("latent, one step", case, time_us(both, iters, profile), 2 * B * ctx * row + 4 * nq * rank * dim, 2.0 * B * ctx * nq * (2 * rank + rot))
        del calls, wcalls
    if not prompts:
        return
    T, npages, ldkv = 4096, 64, nq * (dim + vd)
    bt, pos, slots = torch.arange(npages, **i32).view(1, -1), torch.arange(T, **i32), torch.zeros(T, **i32)
    c = call(T, pos, slots, bt, torch.randn(npages, page, row, device=dev).bfloat16(), *ws[0], 256)
    entries, context = torch.tensor([0, T, 0, 0], **i32), torch.tensor([0, T, 0, 0], **i32)
    tiles = torch.tensor([[0, t] for t in range(0, T, CONTEXT_TILE)], **i32)
    lat, kv = torch.randn(T, row, device=dev).bfloat16(), torch.randn(T, ldkv, device=dev).bfloat16()
    fn = lambda: K.check(lib.bonsai_lay_latent_append(*c.args, 0, T, 0, K.stream()), "latent_append")
    rep.add("latent_append", f"T={T}", time_us(fn, iters, profile), 6 * T * (rank + rot))
    fn = lambda: K.check(lib.bonsai_lay_latent_gather(*c.args, context.data_ptr(), 1, T, lat.data_ptr(), row, K.stream()), "latent_gather")
    rep.add("latent_gather", f"T={T}", time_us(fn, iters, profile), 4 * T * row)
    w, scratch = L.DenseWeight([torch.randn(ldkv, rank).bfloat16()], dev), L.GemmScratch(dev, torch.zeros(1, dtype=torch.int32, device=dev))
    rep.add("linear, bf16 out", f"expand {ldkv}x{rank} T={T}", time_us(lambda: L.linear(w, lat, T, kv, scratch), 10, profile), 2 * T * ldkv + 2 * T * rank + 2 * ldkv * rank,
            2.0 * T * ldkv * rank)
    kv.normal_()
    fn = lambda: K.check(lib.bonsai_lay_latent_prompt(*c.args, entries.data_ptr(), context.data_ptr(), tiles.data_ptr(), len(tiles), kv.data_ptr(), ldkv, lat.data_ptr(), row,
                                                      K.stream()), "latent_prompt")
    rep.add("latent_prompt", f"T={T} heads={nq} {dim}+{rot}, {vd}", time_us(fn, 10, profile), 4 * T * (q_w + g_w) + 2 * T * (ldkv + rot) + 2 * T * g_w,
            2.0 * T * (T + 1) / 2 * nq * (dim + rot + vd))


def bench_experts(rep: Report, width: int, iters: int, profile: bool) -> None:
    """Router and experts; the like kernels are the gate/up, down and residual cases of bench_linear and bench_recurrence."""
    from oxibonsai_b200.models.layered_config import ExpertsSpec, RouterSpec
    from oxibonsai_b200.ops import cuda_ops as K
    from oxibonsai_b200.ops import layered_ops as L
    dev = torch.device("cuda")
    scratch = L.GemmScratch(dev, torch.zeros(1, dtype=torch.int32, device=dev))
    for E, top, ff in ((32, 4, width // 4), (128, 8, width // 4)):
        spec = ExpertsSpec(RouterSpec(E, top, 8, 4, 2.5), ff)
        s = L.ExpertScratch(4096, width, [spec], False, dev)
        logits = torch.randn(4096, E, device=dev)

        def matrix(n, k):
            w = L.DenseWeight([torch.zeros(8, k, dtype=torch.bfloat16)], dev)
            w.n, w.data = E * n, torch.empty(E * n, k, dtype=torch.bfloat16, device=dev).normal_(std=k ** -0.5)
            return w
        r = L.Routing(spec, matrix(2 * ff, width), matrix(width, ff), torch.zeros(E, device=dev), logits, 0, s)
        h = torch.randn(4096, width, device=dev).bfloat16()
        x, y, x16, norm = torch.zeros(4096, width, device=dev), torch.randn(4096, width, device=dev), torch.zeros(4096, width, dtype=torch.bfloat16, device=dev), torch.ones(width, device=dev)
        lib, it = L.lib(), [0]
        for T in (1, 8, 32, 64, 256, 1024, 4096):
            if 8 * T * top < E and T > 8:
                continue
            pairs, few, st, hid = T * top, r.few(T), K.stream, s.hidden[ff]
            xs = None if few else s.sorted

            def route():
                K.check(lib.bonsai_lay_route(*r.call.args, T, h.data_ptr(), h.stride(0), width // 8 if xs is not None else 0, K.ptr(xs), 0 if xs is None else xs.stride(0), st()),
                        "route")
                s.counts.zero_()
            # distinct logits per turn, so that the chosen experts' weights are not in L2 from the turn before
            lists = []
            for _ in range(8):
                logits.normal_()
                route()
                lists.append([t.clone() for t in (s.lists, s.token, s.weight)])
            chosen = sum(int(l[0][E + 1]) for l in lists) / len(lists)
            case, like = f"T={T} {top} of {E} experts, {ff} units, {'few' if few else 'tiles'}", 2 * ff * width

            def route_only():
                K.check(lib.bonsai_lay_route(*r.call.args, T, h.data_ptr(), h.stride(0), width // 8 if xs is not None else 0, K.ptr(xs), 0 if xs is None else xs.stride(0), st()),
                        "route")
                if xs is not None or T > lib.bonsai_lay_route_small(top):
                    L.side_by_side(x, y, r, 0.0, 1, None, None, 1e-6, True)          # a row of it: leaves the counters zero
            rep.add("route", case, time_us(route_only, iters, profile), 4 * T * E + (2 * (T + pairs) * width if xs is not None else 0))

            def up():
                it[0] += 1
                li, tok, wt = lists[it[0] % 8]
                if few:
                    K.check(lib.bonsai_lay_experts_few(r.up.data.data_ptr(), E, 2 * ff, width, h.data_ptr(), width, li.data_ptr(), tok.data_ptr(), wt.data_ptr(), pairs,
                                                       min(E, pairs), min(T, 2 * pairs // E + 8), hid.data_ptr(), ff, 1, float("inf"), 1.0, 0.0, 0.0, st()), "experts_few")
                else:
                    K.check(lib.bonsai_grouped_gemm_bf16(r.up.data.data_ptr(), E, 2 * ff, width, xs.data_ptr(), width, pairs, li.data_ptr(), wt.data_ptr(), hid.data_ptr(), ff, 4,
                                                         float("inf"), 1.0, 0.0, 0.0, int(pairs > 96 * E), scratch.status.data_ptr(), scratch.sms, st()), "grouped_gemm")

            def down():
                it[0] += 1
                li = lists[it[0] % 8][0]
                if few:
                    K.check(lib.bonsai_lay_experts_few(r.down.data.data_ptr(), E, width, ff, hid.data_ptr(), ff, li.data_ptr(), None, None, pairs, min(E, pairs),
                                                       min(T, 2 * pairs // E + 8), s.out32.data_ptr(), s.out32.stride(0), 0, 0.0, 0.0, 0.0, 0.0, st()), "experts_few")
                else:
                    K.check(lib.bonsai_grouped_gemm_bf16(r.down.data.data_ptr(), E, width, ff, hid.data_ptr(), ff, pairs, li.data_ptr(), None, s.out.data_ptr(), s.out.stride(0), 6,
                                                         0.0, 0.0, 0.0, 0.0, int(pairs > 96 * E), scratch.status.data_ptr(), scratch.sms, st()), "grouped_gemm")
            rep.add("experts, gate/up", case, time_us(up, iters, profile), chosen * 2 * like + 2 * (T if few else pairs) * width + 2 * pairs * ff, 4.0 * pairs * ff * width)
            rep.add("experts, down", case, time_us(down, iters, profile), chosen * like + 2 * pairs * ff + (4 if few else 2) * pairs * width, 2.0 * pairs * ff * width)
            r.out = s.out32 if few else s.out
            fn = lambda: L.side_by_side(x, y, r, 0.5, T, x16, norm, 1e-6, True)
            rep.add("side_by_side", case, time_us(fn, iters, profile), (14.0 * T + (4 if few else 2) * pairs) * width)
        del r, s


def bench_recurrence(rep: Report, width: int, iters: int, profile: bool) -> None:
    """The linear recurrences; the like kernels are those of bench_mlstm."""
    from oxibonsai_b200.models.layered import CHUNK, MAX_SEGMENTS, RECURRENCE_COST, WIDE_RECURRENCE_COST, SegmentPlan, plan_segments
    from oxibonsai_b200.ops import cuda_ops as K
    from oxibonsai_b200.ops import layered_ops as L
    dev = torch.device("cuda")
    i32, lib = dict(dtype=torch.int32, device=dev), L.lib()
    H = width // 128
    kinds = {"lightning": dict(h=H, g=H, d=128, e=128, act=1), "retention": dict(h=max(1, width // 256), g=max(1, width // 256), d=256, e=256, rot=256),
             "ssd": dict(h=width // 64, g=max(1, H // 4), d=128, e=64, act=1, taps=4)}
    for name, c in kinds.items():
        h, g, d, e, taps, rot = c["h"], c["g"], c["d"], c["e"], c.get("taps", 0), c.get("rot", 0)
        inner, ch = h * e, h * e + 2 * g * d
        v, k, q, gate, dt = 0, inner, inner + g * d, ch, ch + inner
        ld, ldf = ch + inner + L.round_up(h, 4), lib.bonsai_lay_rec_features_width(h, g, d, e)
        vec = torch.full((h,), 0.99, device=dev)
        conv = (torch.randn(taps, ch, device=dev), torch.randn(ch, device=dev)) if taps else (None, None)
        freq = torch.rand(rot // 2, dtype=torch.float64, device=dev) if rot else None
        scratch = [torch.empty(MAX_SEGMENTS * n, device=dev) for n in (h * d * e, h)]

        def call(T, rows, out, pos, slots):
            S, ring = torch.zeros(rows, h, d, e, device=dev), (torch.zeros(rows, taps, ch, device=dev) if taps else None)
            proj, feat = torch.randn(T, ld, device=dev), torch.zeros(T, ldf, dtype=torch.bfloat16, device=dev)
            return L.MixerCall([proj, None if taps else vec, vec, vec, vec if taps else None, None, *conv, ring, freq, S, pos, slots, torch.arange(rows, **i32), out,
                                feat, *scratch],
                               [ld, q, k, v, gate, dt, 0, out.stride(0), ldf, h, g, d, e, c.get("act", 0), taps, ch if taps else 0, rot, int(name != "lightning")],
                               [1e-6, 1.0, 1.0])
        for B in (1, 8, 64):
            copies = max(2, int(400e6 / (4 * B * h * d * e)) + 1)
            done = name == "retention"
            out = torch.zeros(B, inner, dtype=torch.bfloat16 if done else torch.float32, device=dev)
            calls = [call(B, B, out, torch.full((B,), 5, **i32), torch.arange(B, **i32)) for _ in range(copies)]
            it = [0]

            def step():
                it[0] += 1
                K.check(lib.bonsai_lay_rec_step(*calls[it[0] % copies].args, None, B, 2 if done else 1, 0, 0, K.stream()), "rec_step")
            rep.add("rec_step", f"{name} B={B} heads={h} {d}x{e}", time_us(step, iters, profile), 8.0 * B * h * d * e, 4.0 * B * h * d * e)
            del calls
        for nseq, T in ((1, 4096), (1, 512), (8, 512)):
            rows = nseq * T
            out = torch.zeros(rows, inner, device=dev)
            cl = call(rows, nseq, out, torch.arange(T, **i32).repeat(nseq), torch.arange(nseq, **i32).repeat_interleave(T))
            entries = torch.tensor([[s * T, T, s, 0] for s in range(nseq)], **i32)
            plan = SegmentPlan(h * e // 64, RECURRENCE_COST if d <= 128 else WIDE_RECURRENCE_COST)
            size = plan_segments([T] * nseq, plan, torch.cuda.get_device_properties(dev).multi_processor_count) * CHUNK
            segs = [(s * T + x, min(size, T - x), s, int(x + size >= T)) for s in range(nseq) for x in range(0, T, size)] if size else []
            per = len(segs) // nseq
            sl, pl = torch.tensor(segs or [[0] * 4], **i32), torch.tensor([(s, 0, s * per, per) for s in range(nseq)], **i32)
            case = f"{name} {nseq} x {T} tokens heads={h}/{g} {d}x{e}"
            fn = lambda: K.check(lib.bonsai_lay_rec_features(*cl.args, 0, rows, 0, K.stream()), "rec_features")
            rep.add("rec_features", case, time_us(fn, 10, profile), 6.0 * rows * ch)
            fn = lambda: K.check(lib.bonsai_lay_rec_chunk(*cl.args, entries.data_ptr(), nseq, sl.data_ptr(), len(segs), pl.data_ptr(), K.stream()), "rec_chunk")
            rep.add("rec_chunk", f"{case} segments={len(segs)}", time_us(fn, 10, profile), rows * (2.0 * ch + 4.0 * inner), 4.0 * rows * h * d * e)
            if nseq == 1 and T == 512:
                continue
            act, gates = torch.zeros(rows, inner, dtype=torch.bfloat16, device=dev), torch.randn(rows, ld, device=dev)
            parts = {"lightning": 1, "retention": h, "ssd": g}[name]
            fn = lambda: L.gated_norm(out, 0, gates, gate, None, 1e-6, rows, parts, inner // parts, act, "silu", name == "ssd")
            rep.add("gated_norm", f"{name} T={rows} parts={parts}", time_us(fn, iters, profile), 10.0 * rows * inner)
    for T in (1, 64, 4096):
        x, y, w = torch.randn(T, width, device=dev), torch.randn(T, width, device=dev), torch.ones(width, device=dev)
        x16 = torch.zeros(T, width, dtype=torch.bfloat16, device=dev)
        rep.add("norm_add, next norm", f"T={T} width={width}", time_us(lambda: L.norm_add(x, y, w, 1e-6, T, x16, w), iters, profile), 14.0 * T * width)


def bench_mlstm(rep: Report, width: int, iters: int, profile: bool) -> None:
    from oxibonsai_b200.ops import cuda_ops as K
    from oxibonsai_b200.ops import layered_ops as L
    dev = torch.device("cuda")
    H, d, e = max(2, width // 512), 256, 512
    cols = [0, H * d, 2 * H * d, 2 * H * d + H * e, 2 * H * d + 2 * H * e, 2 * H * d + 2 * H * e + 4]
    ld = cols[-1] + 8
    i32 = dict(dtype=torch.int32, device=dev)
    bias, norm = torch.zeros(H + 4, device=dev), torch.ones(H * e, device=dev)

    from oxibonsai_b200.models.layered import CHUNK, MAX_SEGMENTS, MLSTM_COST, SegmentPlan, plan_segments
    scratch = [torch.empty(MAX_SEGMENTS * n, device=dev) for n in (H * d * e, H * d * e // 64, H * e // 64, H * e // 32)]

    def call(T, rows, out, states, pos):
        proj = torch.randn(T, ld, device=dev)
        S, n, m = states
        return L.MixerCall([proj, bias, bias + 4, norm, S, n, m, pos, torch.arange(rows, **i32), torch.arange(rows, **i32), out, *scratch],
                           [ld, *cols, out.stride(0), H, d, e], [15.0, 1e-6, 1e-6, d ** -0.5])
    state = lambda rows: (torch.zeros(rows, H, d, e, device=dev), torch.zeros(rows, H, e // 64, d, device=dev), torch.zeros(rows, H, e // 64, device=dev))
    for B in (1, 8, 64):
        copies = max(2, int(400e6 / (4 * B * H * d * e)) + 1)
        out = torch.zeros(B, H * e, dtype=torch.bfloat16, device=dev)
        calls = [call(B, B, out, state(B), torch.full((B,), 5, **i32)) for _ in range(copies)]
        it = [0]

        def step():
            it[0] += 1
            K.check(L.lib().bonsai_lay_mlstm_step(*calls[it[0] % copies].args, None, B, 1, K.stream()), "mlstm_step")
        rep.add("mlstm_step", f"B={B} heads={H} {d}x{e}", time_us(step, iters, profile), 8.0 * B * H * d * e, 4.0 * B * H * d * e)
        del calls
    for nseq, T in ((1, 4096), (1, 512), (8, 512)):
        rows = nseq * T
        out = torch.zeros(rows, H * e, device=dev)
        c = call(rows, nseq, out, state(nseq), torch.zeros(nseq, **i32))
        entries = torch.tensor([[s * T, T, s, 0] for s in range(nseq)], **i32)
        size = plan_segments([T] * nseq, SegmentPlan(H * e // 64, MLSTM_COST), torch.cuda.get_device_properties(dev).multi_processor_count) * CHUNK
        segs = [(s * T + x, min(size, T - x), s, int(x + size >= T)) for s in range(nseq) for x in range(0, T, size)] if size else []
        per = len(segs) // nseq
        sl = torch.tensor(segs or [[0] * 4], **i32)
        pl = torch.tensor([(s, 0, s * per, per) for s in range(nseq)], **i32)
        fn = lambda: K.check(L.lib().bonsai_lay_mlstm_chunk(*c.args, entries.data_ptr(), nseq, sl.data_ptr(), len(segs), pl.data_ptr(), K.stream()), "mlstm_chunk")
        # the recurrence's own products (k v^T and S^T q) against one pass over q, k, v and o
        rep.add("mlstm_chunk", f"{nseq} x {T} tokens heads={H} {d}x{e} segments={len(segs)}", time_us(fn, 10, profile), 4.0 * rows * H * (2 * d + 2 * e), 4.0 * rows * H * d * e)
        act = torch.zeros(rows, H * e, dtype=torch.bfloat16, device=dev)
        gate = torch.randn(rows, ld, device=dev)
        rep.add("gated_head_norm", f"T={rows}", time_us(lambda: L.gated_norm(out, 0, gate, 0, norm, 1e-6, rows, H, e, act), iters, profile), 10.0 * rows * H * e)
    for T in (1, 64, 4096):
        x, y, w = torch.randn(T, width, device=dev), torch.randn(T, width, device=dev), torch.ones(width, device=dev)
        x16 = torch.zeros(T, width, dtype=torch.bfloat16, device=dev)
        rep.add("norm_add", f"T={T} width={width}", time_us(lambda: L.norm_add(x, y, w, 1e-6, T, x16), iters, profile), 14.0 * T * width)


class BenchRows:
    """Rows of ``nseq`` sequences, single tokens at position ``pos`` or portions of ``T`` tokens, with the lists of a step."""

    def __init__(self, nseq: int, T: int, pos: int = 0):
        from oxibonsai_b200.models.layered import StepShape
        from oxibonsai_b200.ops import layered_ops as L
        i32, rows, tile = dict(dtype=torch.int32, device="cuda"), nseq * T, L.lib().bonsai_lay_conv_rows()
        self.tokens, self.rows = torch.zeros(rows, **i32), rows
        self.positions = torch.arange(T, **i32).repeat(nseq) + pos
        self.slots, self.state = torch.arange(nseq, **i32).repeat_interleave(T), torch.arange(nseq, **i32)
        if T == 1:
            self.shape = StepShape(rows, rows, rows)
            return
        self.entries = torch.tensor([[s * T, T, s, pos] for s in range(nseq)], **i32)
        self.tiles = torch.tensor([[s, t] for s in range(nseq) for t in range(0, T, tile)], **i32)
        self.shape = StepShape(rows, 0, 0, nseq, self.entries.data_ptr(), {tile: (self.tiles.data_ptr(), len(self.tiles))})


def bench_differential(rep: Report, width: int, iters: int, profile: bool) -> None:
    """Two maps of 64 dimensions over values of 128; the like kernels are those of bench_capped_attention and bench_rotary."""
    from oxibonsai_b200.ops import cuda_ops as K
    from oxibonsai_b200.ops import layered_ops as L
    dev = torch.device("cuda")
    nq, nkv, hd, page = width // 128, max(1, width // 512), 128, 64
    i32 = dict(dtype=torch.int32, device=dev)
    ld = (2 * nq + 2 * nkv) * hd
    rot, norm, bias = torch.randn(4096, 32, 2, device=dev), torch.ones(64, device=dev), torch.zeros(nq * hd, device=dev)

    def call(proj, pos, slots, bt, k, v, out):
        return L.MixerCall([proj, norm, norm, None, pos, slots, bt, k, None, v, out, None, rot, bias, bias, bias],
                           [ld, 0, nq * hd, (nq + nkv) * hd, (nq + 2 * nkv) * hd, nq * hd, nq, nkv, 64, hd, bt.shape[1], page, 0, 0, 1, 64, 1, 8192, 2, 1],
                           [1e-6, 0.125, 1.0, 0.0, 0.0, 1.0, 0.6, 0.5])
    per_pair = 2.0 * nq * (2 * 64 + 2 * hd)
    for B, ctx in ((1, 4096), (8, 4096), (64, 1024)):
        npages = ctx // page
        copies = max(2, int(300e6 / (4 * B * ctx * nkv * hd)) + 1)
        pools = [[torch.randn(B * npages, nkv, page, hd, device=dev).bfloat16() for _ in range(2)] for _ in range(copies)]
        bt = torch.arange(B * npages, **i32).view(B, npages)
        pos, slots, proj = torch.full((B,), ctx - 1, **i32), torch.arange(B, **i32), torch.randn(B, ld, device=dev)
        out = torch.zeros(B, nq * hd, dtype=torch.bfloat16, device=dev)
        calls = [call(proj, pos, slots, bt, *p, out) for p in pools]
        it, split = [0], 1
        while split < 8 and B * nkv * split * 2 <= 160:
            split *= 2

        def ours():
            it[0] += 1
            K.check(L.lib().bonsai_lay_attn_decode(*calls[it[0] % copies].args, B, split, K.stream()), "attn_decode")
        rep.add("attn_decode, two maps", f"B={B} ctx={ctx} heads={nq}/{nkv}", time_us(ours, iters, profile), 4 * B * ctx * nkv * hd, per_pair * B * ctx)
    T, npages = 4096, 64
    k, v = (torch.randn(npages, nkv, page, hd, device=dev).bfloat16() for _ in range(2))
    bt, pos, slots = torch.arange(npages, **i32).view(1, -1), torch.arange(T, **i32), torch.zeros(T, **i32)
    proj, out = torch.randn(T, ld, device=dev), torch.zeros(T, nq * hd, dtype=torch.bfloat16, device=dev)
    entries = torch.tensor([0, T, 0, 0], **i32)
    tiles = torch.tensor([[0, t] for t in range(0, T, 64 // (nq // nkv))], **i32)
    c = call(proj, pos, slots, bt, k, v, out)
    fn = lambda: K.check(L.lib().bonsai_lay_attn_prompt(*c.args, entries.data_ptr(), tiles.data_ptr(), len(tiles), K.stream()), "attn_prompt")
    rep.add("attn_prompt, two maps", f"T={T} heads={nq}/{nkv}", time_us(fn, 10, profile), 4 * T * ld + 4 * T * nkv * hd + 2 * T * nq * hd, per_pair * T * (T + 1) / 2)
    fn = lambda: K.check(L.lib().bonsai_lay_attn_append(*c.args, 0, T, 0, K.stream()), "attn_append")
    rep.add("attn_append, two maps", f"T={T}", time_us(fn, iters, profile), 12 * T * nkv * hd)


def bench_scans(rep: Report, width: int, iters: int, profile: bool) -> None:
    """minGRU, the selective scan and the convolutions; the like kernels are those of bench_recurrence."""
    from oxibonsai_b200.models.layered import CHUNK, MAX_SEGMENTS, SCAN_COST, SegmentPlan, plan_segments
    from oxibonsai_b200.ops import cuda_ops as K
    from oxibonsai_b200.ops import layered_ops as L
    dev, lib = torch.device("cuda"), L.lib()
    sms, W, N, R = torch.cuda.get_device_properties(dev).multi_processor_count, width, 16, width // 16
    inner, i32, it = 2 * width, dict(dtype=torch.int32, device=dev), [0]
    vec = torch.zeros(inner, device=dev)

    def turn(calls, fn):
        def run():
            it[0] += 1
            fn(calls[it[0] % len(calls)].args)
        return run

    def gru(rows):
        proj, out = torch.randn(rows.rows, 3 * W, device=dev), torch.zeros(rows.rows, W, dtype=torch.bfloat16, device=dev)
        return L.MixerCall([proj, vec, vec, torch.zeros(len(rows.state), W, device=dev), rows.positions, rows.slots, rows.state, out], [3 * W, 0, W, 2 * W, W, W], [])
    scratch = [torch.empty(MAX_SEGMENTS * inner * n, device=dev) for n in (N, 1)]
    A = -torch.rand(inner, N, device=dev)

    def scan(rows):
        T = rows.rows
        proj, bc, dt = torch.randn(T, 2 * inner, device=dev), torch.randn(T, R + 2 * N, device=dev), torch.randn(T, inner, device=dev)
        x, out = (torch.randn(T, inner, device=dev).bfloat16() for _ in range(2))
        return L.MixerCall([proj, bc, dt, x, vec, A, vec, torch.zeros(len(rows.state), inner, N, device=dev), rows.positions, rows.slots, rows.state, out, *scratch],
                           [2 * inner, inner, R + 2 * N, R, R + N, inner, inner, inner, inner, N], [])
    for B in (1, 8, 64):
        rows, copies = BenchRows(B, 1, 5), 2 + int(300e6 / (B * inner * (8 * N + 14)))
        rep.add("gru_step", f"B={B} width={W}", time_us(turn([gru(rows) for _ in range(copies)], lambda a: K.check(lib.bonsai_lay_gru_step(*a, B, 0, K.stream()), "gru_step")),
                                                        iters, profile), 22.0 * B * W)
        rep.add("scan_step", f"B={B} {inner} x {N}", time_us(turn([scan(rows) for _ in range(copies)], lambda a: K.check(lib.bonsai_lay_scan_step(*a, B, 0, K.stream()), "scan_step")),
                                                             iters, profile), B * inner * (8.0 * N + 12) + 4.0 * inner * N)
        conv = lambda c: L.Conv(torch.randn(B, c, device=dev), 0, c, torch.randn(4, c, device=dev), vec, torch.zeros(B, 4, c, device=dev), rows, rows.state,
                                torch.zeros(B, c, dtype=torch.bfloat16, device=dev), silu=True)
        convs = [conv(inner) for _ in range(copies)]

        def run_conv():
            it[0] += 1
            convs[it[0] % copies](rows.shape)
        rep.add("conv, silu", f"B={B} channels={inner}", time_us(run_conv, iters, profile), 22.0 * B * inner)
    for nseq, T in ((1, 4096), (1, 512), (8, 512)):
        rows, n = BenchRows(nseq, T), nseq * T
        copies = 1 + int(300e6 / (14.0 * n * W))
        cluster, ctas = 1, nseq * -(-W // 32)
        while cluster < 8 and 2 * cluster * ctas <= 4 * sms and 2 * cluster * lib.bonsai_lay_gru_tokens() <= T:
            cluster *= 2
        fn = lambda a: K.check(lib.bonsai_lay_gru_scan(*a, rows.shape.entries, nseq, cluster, 0, K.stream()), "gru_scan")
        rep.add("gru_scan", f"{nseq} x {T} tokens width={W} cluster={cluster}", time_us(turn([gru(rows) for _ in range(copies)], fn), 10, profile), 14.0 * n * W)
        plan = SegmentPlan(-(-inner // lib.bonsai_lay_scan_channels(N)), SCAN_COST)
        size = plan_segments([T] * nseq, plan, sms) * CHUNK
        for size in sorted({0, size}):
            if size and nseq * -(-T // size) > MAX_SEGMENTS or size >= T:
                continue
            segs = [(s * T + x, min(size, T - x), s, int(x + size >= T)) for s in range(nseq) for x in range(0, T, size)] if size else []
            per = len(segs) // nseq
            sl, pl = torch.tensor(segs or [[0] * 4], **i32), torch.tensor([(s, 0, s * per, per) for s in range(nseq)], **i32)
            fn = lambda a: K.check(lib.bonsai_lay_scan(*a, rows.shape.entries, nseq, sl.data_ptr(), len(segs), pl.data_ptr(), 0, K.stream()), "scan")
            rep.add("scan", f"{nseq} x {T} tokens {inner} x {N} segments={len(segs)}", time_us(turn([scan(rows)], fn), 10, profile), n * (12.0 * inner + 8 * N))
        if n < 4096 or nseq > 1:
            continue
        for c, silu in ((W, False), (inner, True)):
            x, out = torch.randn(n, c, device=dev), torch.zeros(n, c, dtype=torch.bfloat16, device=dev)
            conv = L.Conv(x, 0, c, torch.randn(4, c, device=dev), vec if silu else None, torch.zeros(nseq, 4, c, device=dev), rows, rows.state, out, add=not silu, silu=silu)
            rep.add("conv" + (", silu" if silu else ", added"), f"T={n} channels={c}", time_us(lambda: conv(rows.shape), iters, profile), 6.0 * n * c)
        bc, low = torch.randn(n, R + 2 * N, device=dev), torch.zeros(n, L.round_up(R, 128), dtype=torch.bfloat16, device=dev)
        rep.add("narrow", f"T={n} columns={R}", time_us(lambda: L.narrow(bc, 0, R, n, low), iters, profile), 6.0 * n * R)
        scratch2 = L.GemmScratch(dev, torch.zeros(1, dtype=torch.int32, device=dev))
        for rows_, k in ((R + 2 * N, inner), (inner, R)):
            for T2 in (1, 64, n):
                w = L.DenseWeight([torch.randn(rows_, k).bfloat16()], dev)
                x, out = torch.randn(n, w.kp, device=dev).bfloat16(), torch.zeros(n, rows_, device=dev)
                rep.add("linear", f"{rows_}x{k} T={T2}", time_us(lambda: L.linear(w, x, T2, out, scratch2), iters, profile), 2.0 * rows_ * k + T2 * (2.0 * k + 4 * rows_), 2.0 * T2 * rows_ * k)


def bench_row_steps(rep: Report, width: int, iters: int, profile: bool) -> None:
    """The general row step, the gelu gate, the capped head and the softmax router; the like kernels are norm_add, side_by_side, the gated
    and the plain projections and the sigmoid router."""
    from oxibonsai_b200.models.layered_config import ExpertsSpec, RouterSpec, gelu_mlp
    from oxibonsai_b200.ops import layered_ops as L
    dev, W = torch.device("cuda"), width
    scratch = L.GemmScratch(dev, torch.zeros(1, dtype=torch.int32, device=dev))
    w = torch.ones(W, device=dev)
    for T in (1, 8, 64, 4096):
        rows = BenchRows(T, 1, 9) if T < 4096 else BenchRows(1, T)
        x, y, h = torch.randn(T, W, device=dev), torch.randn(T, W, device=dev), torch.zeros(T, W, dtype=torch.bfloat16, device=dev)
        conv, n32 = (torch.randn(4, W, device=dev), torch.zeros(len(rows.state), 4, W, device=dev)), torch.zeros(T, W, device=dev)
        common = dict(eps=1e-6, groups=4, mult=0.5, y=y, w=w, next_norm=w)
        plain = L.RowStep(x, h, rows, rows.state, **common)
        rep.add("row_step", f"T={T} width={W}", time_us(lambda: plain(T, rows.shape), iters, profile), 14.0 * T * W)
        full = L.RowStep(x, h, rows, rows.state, conv=conv, n32=n32, **common)
        rep.add("row_step, convolution", f"T={T} width={W}", time_us(lambda: full(T, rows.shape), iters, profile), (14.0 + (16 if T < 4096 else 0)) * T * W)
        spec = ExpertsSpec(RouterSpec(32, 4, softmax=True, normalized=False, corrected=False), 64)
        s, logits = L.ExpertScratch(T, W, [spec], False, dev), torch.randn(T, 36, device=dev)
        r = L.Routing(spec, L.DenseWeight([torch.zeros(64 * 32, 128).bfloat16()] * 2, dev, interleave=True), L.DenseWeight([torch.zeros(8, 128).bfloat16()], dev), None, logits, 0, s)
        s.at.copy_(torch.randperm(4 * T, device=dev).int())
        step = L.RowStep(x, h, rows, rows.state, gate=logits[:, 32:], **common)
        rep.add("row_step, experts", f"T={T} width={W}", time_us(lambda: step(T, rows.shape, r), iters, profile), 22.0 * T * W)
    g = gelu_mlp(3 * W)
    for T in (1, 64, 4096):
        for name, n, act in (("gate_up, gelu", 6 * W, L.Glu(g.limit, g.alpha, g.offset, g.cubic)), ("head, capped", 32000, L.SoftCap(30.0))):
            copies = 3
            ws = []
            for _ in range(copies):
                m = L.DenseWeight([torch.zeros(8, W, dtype=torch.bfloat16)], dev)
                m.n, m.data = n, torch.randn(n, W, device=dev).bfloat16()
                ws.append(m)
            h = torch.randn(T, W, device=dev).bfloat16()
            out = torch.empty(T, n // 2, dtype=torch.bfloat16, device=dev) if "gate" in name else torch.empty(T, n, device=dev)
            it = [0]

            def run():
                it[0] += 1
                L.linear(ws[it[0] % copies], h, T, out, scratch, act)
            rep.add("linear", f"{name} {n}x{W} T={T}", time_us(run, iters, profile), 2.0 * n * W + 2.0 * T * W + out.numel() * out.element_size(), 2.0 * T * n * W)


# ---- whole models ---------------------------------------------------------------------------------------------------------------------
SIZES = {"s": dict(width=1024, repeats=3), "m": dict(width=2048, repeats=4), "l": dict(width=4096, repeats=4)}


def _event_ms(fn, n: int) -> float:
    e0, e1 = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
    torch.cuda.synchronize()
    e0.record()
    for _ in range(n):
        fn()
    e1.record()
    torch.cuda.synchronize()
    return e0.elapsed_time(e1) / n


def measure_layered(path: str, steps: int, warmup: int, prompt: int, batches) -> dict:
    from oxibonsai_b200.runtime import EngineBuilder
    eng = EngineBuilder().model_path(path).preset("greedy").max_seq_len(prompt + 3 * (steps + warmup) + 64).max_batch(max(batches)).kv_cache("bf16").build()
    r, vocab = eng.runner, eng.config.vocab
    toks = torch.randint(0, vocab, (prompt,), generator=torch.Generator().manual_seed(1)).tolist()
    res = {"weight_GB": round(eng.weights.packed_bytes / 1e9, 3), "launches_per_step": r.kernel_launches(1)}
    for b in range(max(batches)):
        eng.reserve(b, prompt + 3 * (steps + warmup) + 8)
    for _ in range(3):
        eng.prefill(toks, 0)
    ms = _event_ms(lambda: eng.prefill(toks, 0), 5)
    res[f"prefill_{prompt}_tok_s"] = round(prompt / ms * 1e3)
    for b in range(1, max(batches)):
        eng.prefill(toks, b)
    for B in batches:
        r.positions[:B].fill_(prompt)
        for _ in range(warmup):
            r.step(B)
        ms = _event_ms(lambda: r.step(B), steps)
        res[f"decode_b{B}_tok_s"], res[f"decode_b{B}_ms"] = round(B / ms * 1e3, 1), round(ms, 4)
    r.check_status()
    return res


def measure_generic(path: str, steps: int, warmup: int, prompt: int, batches) -> dict:
    from oxibonsai_b200.runtime.engine import GenericFormatEngine
    eng = GenericFormatEngine(path, max_seq_len=prompt + 3 * (steps + warmup) + 64, max_batch=max(batches))
    e = eng._eng
    toks = torch.randint(0, eng.config.vocab, (prompt,), generator=torch.Generator().manual_seed(1)).tolist()
    res = {"weight_GB": round(eng.model_info()["weight_bytes"] / 1e9, 3), "launches_per_step": e.kernel_launches_per_step(1)}
    for b in range(max(batches)):
        eng.begin_sequence(toks, prompt + 3 * (steps + warmup), b)
    dt = torch.tensor(toks, dtype=torch.int32, device="cuda")
    for _ in range(3):
        e.prefill(dt, 0, 0)
    ms = _event_ms(lambda: e.prefill(dt, 0, 0), 5)
    res[f"prefill_{prompt}_tok_s"] = round(prompt / ms * 1e3)
    for b in range(1, max(batches)):
        e.prefill(dt, 0, b)
    for B in batches:
        e.pos[:B].fill_(prompt)
        for _ in range(warmup):
            e.step(B)
        ms = _event_ms(lambda: e.step(B), steps)
        res[f"decode_b{B}_tok_s"], res[f"decode_b{B}_ms"] = round(B / ms * 1e3, 1), round(ms, 4)
    return res


def run_kekevik(sizes, steps: int = 64, warmup: int = 5, prompt: int = 2048, batches=(1, 8, 64), log=sys.stdout) -> list[dict]:
    """Kekevik beside Keripel of the same width with as many layers as bring it to the same parameter count."""
    rows = []
    for size in sizes:
        width, repeats = SIZES[size]["width"], max(1, SIZES[size]["repeats"] // 2)
        row = {"size": size, "width": width}
        for name, make in (("kekevik", kekevik), ("keripel", keripel)):
            with tempfile.TemporaryDirectory() as d:
                if name == "keripel":
                    count = lambda n: write_design(os.path.join(d, "m"), keripel(width, n))
                    one, two = count(1), count(2)
                    repeats = max(1, round((row["kekevik_params_M"] * 1e6 - one) / (two - one)) + 1)
                cfg = make(width, repeats)
                params = write_design(os.path.join(d, "m"), cfg)
                row[f"{name}_layers"], row[f"{name}_params_M"] = len(cfg["layers"]), round(params / 1e6)
                row[name] = measure_layered(os.path.join(d, "m"), steps, warmup, prompt, batches)
            torch.cuda.empty_cache()
        rows.append(row)
        print(json.dumps(row), file=log, flush=True)
    return rows


def active_params(cfg: dict) -> int:
    """Parameters a token uses: all but the experts that are not chosen."""
    from oxibonsai_b200.models.registry import ARCHITECTURES
    c = ARCHITECTURES[cfg["architecture"]](cfg, "")
    idle = sum(3 * c.experts(i).ff * c.width * (c.experts(i).router.experts - c.experts(i).router.top) for i in c.expert_layers)
    return c.param_count() - idle


def run_kutepel(sizes, steps: int = 64, warmup: int = 5, prompt: int = 2048, batches=(1, 8, 64), log=sys.stdout) -> list[dict]:
    """Kutepel beside Kekevik of the same width with as many layers as bring it to the same parameter count, and to the count that a
    token of Kutepel uses."""
    rows = []
    for size in sizes:
        width, repeats = SIZES[size]["width"], {"s": 1, "m": 1, "l": 1}[size]
        cfg = kutepel(width, repeats)
        row = {"size": size, "width": width, "kutepel_layers": len(cfg["layers"]), "active_params_M": round(active_params(cfg) / 1e6)}
        with tempfile.TemporaryDirectory() as d:
            row["params_M"] = round(write_design(os.path.join(d, "m"), cfg) / 1e6)
            row["kutepel"] = measure_layered(os.path.join(d, "m"), steps, warmup, prompt, batches)
        torch.cuda.empty_cache()
        for name, target in (("kekevik", row["params_M"]), ("kekevik_active", row["active_params_M"])):
            with tempfile.TemporaryDirectory() as d:
                count = lambda n: write_design(os.path.join(d, "m"), kekevik(width, n))
                one, two = count(1), count(2)
                cfg = kekevik(width, max(1, round((target * 1e6 - one) / (two - one)) + 1))
                params = write_design(os.path.join(d, "m"), cfg)
                row[f"{name}_layers"], row[f"{name}_params_M"] = len(cfg["layers"]), round(params / 1e6)
                row[name] = measure_layered(os.path.join(d, "m"), steps, warmup, prompt, batches)
            torch.cuda.empty_cache()
        rows.append(row)
        print(json.dumps(row), file=log, flush=True)
    return rows


def used_params(cfg: dict) -> int:
    """Parameters a token uses, those of a loop as often as it runs."""
    from oxibonsai_b200.models.registry import ARCHITECTURES
    c = ARCHITECTURES[cfg["architecture"]](cfg, "")
    size = lambda prefix: sum(torch.Size(s).numel() for n, s in c.tensor_shapes().items() if n.startswith(prefix))
    idle = lambda i: 3 * c.experts(i).ff * c.width * (c.experts(i).router.experts - c.experts(i).router.top) if i in c.expert_layers else 0
    return size("head") + sum(size(f"l{r.layer}.") - idle(r.layer) for r in c.runs)


def run_naforax(sizes, steps: int = 64, warmup: int = 5, prompt: int = 2048, batches=(1, 8, 64), log=sys.stdout) -> list[dict]:
    """Naforax beside Kekevik of the same width with as many layers as bring it to the same parameter count, and to the count that a
    token of Naforax uses (its loop counted as often as it runs)."""
    rows = []
    for size in sizes:
        width = SIZES[size]["width"]
        cfg = naforax(width, 1)
        row = {"size": size, "width": width, "naforax_layers": len(cfg["layers"]), "used_params_M": round(used_params(cfg) / 1e6)}
        with tempfile.TemporaryDirectory() as d:
            row["params_M"] = round(write_design(os.path.join(d, "m"), cfg) / 1e6)
            row["naforax"] = measure_layered(os.path.join(d, "m"), steps, warmup, prompt, batches)
        torch.cuda.empty_cache()
        for name, target in (("kekevik", row["params_M"]), ("kekevik_used", row["used_params_M"])):
            with tempfile.TemporaryDirectory() as d:
                count = lambda n: write_design(os.path.join(d, "m"), kekevik(width, n))
                one, two = count(1), count(2)
                other = kekevik(width, max(1, round((target * 1e6 - one) / (two - one)) + 1))
                params = write_design(os.path.join(d, "m"), other)
                row[f"{name}_layers"], row[f"{name}_params_M"] = len(other["layers"]), round(params / 1e6)
                row[name] = measure_layered(os.path.join(d, "m"), steps, warmup, prompt, batches)
            torch.cuda.empty_cache()
        rows.append(row)
        print(json.dumps(row), file=log, flush=True)
    return rows


def run_models(sizes, steps: int = 64, warmup: int = 5, prompt: int = 2048, batches=(1, 8, 64), log=sys.stdout) -> list[dict]:
    from oxibonsai_b200.cli import requantize_gguf
    from oxibonsai_b200.core import Qwen3Config, write_synthetic_gguf
    rows = []
    for size in sizes:
        cfg = keripel(**SIZES[size])
        width = cfg["width"]
        with tempfile.TemporaryDirectory() as d:
            params = write_design(os.path.join(d, "design"), cfg)
            ours = measure_layered(os.path.join(d, "design"), steps, warmup, prompt, batches)
        torch.cuda.empty_cache()
        heads, kv, inter, vocab = width // 128, max(1, width // 512), 3 * width, cfg["vocab"]
        per_layer = width * (heads + 2 * kv) * 128 + heads * 128 * width + 3 * width * inter
        layers = max(1, round((params - vocab * width) / per_layer))
        with tempfile.TemporaryDirectory() as d:
            packed, path = os.path.join(d, "packed.gguf"), os.path.join(d, "generic.gguf")
            write_synthetic_gguf(packed, Qwen3Config(hidden=width, inter=inter, layers=layers, heads=heads, kv_heads=kv, head_dim=128, vocab=vocab,
                                                   context=8192, name="generic"), tied=True, seed=1)
            requantize_gguf(packed, path, "f16")
            like = measure_generic(path, steps, warmup, prompt, batches)
        torch.cuda.empty_cache()
        row = {"size": size, "width": width, "design_layers": len(cfg["layers"]), "generic_layers": layers, "params_M": round(params / 1e6),
               "generic_params_M": round((layers * per_layer + vocab * width) / 1e6), "design": ours, "generic_f16": like}
        rows.append(row)
        print(json.dumps(row), file=log, flush=True)
    return rows


def main() -> None:
    ap = argparse.ArgumentParser()
    ap.add_argument("case", choices=["kernels", "models"])
    ap.add_argument("--width", type=int, default=4096)
    ap.add_argument("--only", default="linear,attention,mlstm,capped,recurrence,rotary,latent,experts,differential,scans,rows")
    ap.add_argument("--design", choices=["keripel", "kekevik", "kutepel", "naforax"], default="naforax")
    ap.add_argument("--iters", type=int, default=40)
    ap.add_argument("--sizes", default="s,m,l")
    ap.add_argument("--profile", action="store_true", help="a few eager launches per case, for captures under a profiler")
    a = ap.parse_args()
    torch.cuda.set_device(0)
    if a.case == "models":
        {"keripel": run_models, "kekevik": run_kekevik, "kutepel": run_kutepel, "naforax": run_naforax}[a.design](a.sizes.split(","))
        return
    rep = Report()
    for name, fn in (("linear", bench_linear), ("attention", bench_attention), ("mlstm", bench_mlstm), ("capped", bench_capped_attention),
                     ("recurrence", bench_recurrence), ("rotary", bench_rotary), ("latent", bench_latent), ("experts", bench_experts),
                     ("differential", bench_differential), ("scans", bench_scans), ("rows", bench_row_steps)):
        if name in a.only.split(","):
            fn(rep, a.width, a.iters, a.profile)
            torch.cuda.empty_cache()             # buffers cut out of a former bench's blocks were slower to read by a quarter


if __name__ == "__main__":
    main()
