"""Plain, slow implementation of the layer-list decoders, one function per mechanism: what the GPU path is compared with.

Everything runs on the CPU in the dtype of the tensors it is given (float64 in the tests), one whole sequence at a time,
without a cache, a batch or a chunk.  ``w`` is a dict of tensors by checkpoint name; ``cfg`` is the parsed ``config.json``.
It shares no code with the package.
"""
import math

import torch


def rms(x, eps):
    return x / torch.sqrt((x * x).mean(-1, keepdim=True) + eps)


def rms_norm(x, weight, eps):
    return rms(x, eps) * weight


def linear(x, weight):
    return x @ weight.T


# ---- attention ------------------------------------------------------------------------------------------------------------
def alibi_slope(head, heads):
    return 2.0 ** (-8.0 * (head + 1) / heads)


def visible(i, j, size, keep_first):
    """May position ``i`` see position ``j``: the last ``size`` positions (its own included) and the first ``keep_first`` ones."""
    return j <= i and (i - j < size or j < keep_first)


def window_mask(n, size, keep_first):
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & ((i - j < size) | (j < keep_first))


def softmax_attention(q, k, v, scale, slope, mask):
    """One head: q [n, d], k [n, d], v [n, e]; a linear distance bias is taken off the scores before the softmax."""
    n = q.shape[0]
    dist = (torch.arange(n)[:, None] - torch.arange(n)[None, :]).to(q.dtype)
    s = (q @ k.T) * scale - slope * dist
    return torch.softmax(s.masked_fill(~mask, float("-inf")), dim=-1) @ v


def head_gate(o, h, w_g):
    """o [n, heads, e] times one sigmoid per token and head."""
    return o * torch.sigmoid(linear(h, w_g))[:, :, None]


def attention_mixer(h, w, p, m, eps):
    """Grouped-query attention whose values are the un-normalised keys."""
    n, H, G, d = h.shape[0], m["heads"], m["kv_heads"], m["dim"]
    q = linear(h, w[p + "q"]).view(n, H, d)
    k = linear(h, w[p + "k"]).view(n, G, d)
    v = k
    q, k = rms_norm(q, w[p + "q.norm"], eps), rms_norm(k, w[p + "k.norm"], eps)
    mask = window_mask(n, m["mask"]["size"], m["mask"]["keep_first"])
    o = torch.stack([softmax_attention(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], m["scale"], alibi_slope(a, H), mask) for a in range(H)], dim=1)
    return linear(head_gate(o, h, w[p + "g"]).reshape(n, H * m["vdim"]), w[p + "o"])


# ---- matrix-memory recurrence -----------------------------------------------------------------------------------------------
def soft_cap(x, cap):
    return cap * torch.tanh(x / cap)


def log_gates(h, w, p, cap):
    """Log input and log forget gates, [n, heads] each."""
    i = soft_cap(linear(h, w[p + "i"]) + w[p + "i.b"], cap)
    f = soft_cap(linear(h, w[p + "f"]) + w[p + "f.b"], cap)
    return i, torch.nn.functional.logsigmoid(f)


def matrix_memory(q, k, v, i, f, state=None):
    """One head, token by token: q, k [n, d], v [n, e], i, f [n].  Returns (o [n, e], (S, n, m))."""
    d, e = q.shape[1], v.shape[1]
    S, nrm, mx = (torch.zeros(d, e, dtype=q.dtype), torch.zeros(d, dtype=q.dtype), torch.zeros((), dtype=q.dtype)) if state is None else state
    out = []
    for t in range(q.shape[0]):
        m_new = torch.maximum(f[t] + mx, i[t])
        a, b = torch.exp(f[t] + mx - m_new), torch.exp(i[t] - m_new)
        S = a * S + b * torch.outer(k[t], v[t])
        nrm = a * nrm + b * k[t]
        mx = m_new
        out.append((S.T @ q[t]) / (torch.maximum((nrm @ q[t]).abs(), torch.exp(-mx)) + 1e-6))
    return torch.stack(out), (S, nrm, mx)


def mlstm_mixer(h, w, p, m, eps):
    n, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q = linear(h, w[p + "q"]).view(n, H, d) * d ** -0.5
    k = linear(h, w[p + "k"]).view(n, H, d)
    v = linear(h, w[p + "v"]).view(n, H, e)
    i, f = log_gates(h, w, p, m["gate_cap"])
    o = torch.stack([matrix_memory(q[:, a], k[:, a], v[:, a], i[:, a], f[:, a])[0] for a in range(H)], dim=1)
    o = rms(o, eps).reshape(n, H * e) * w[p + "norm"]
    return linear(o * torch.sigmoid(linear(h, w[p + "g"])), w[p + "o"])


# ---- feed-forward and the whole model ------------------------------------------------------------------------------------------
def clamped_glu(g, u, limit):
    g, u = torch.clamp(g, max=limit), torch.clamp(u, -limit, limit)
    return g * torch.sigmoid(1.702 * g) * (u + 1)


def dense_ff(x, w, p, limit):
    return linear(clamped_glu(linear(x, w[p + "gate"]), linear(x, w[p + "up"]), limit), w[p + "down"])


MIXERS = {"attention": attention_mixer, "mlstm": mlstm_mixer}


def forward(cfg, w, tokens, keep_layers=False):
    """Logits [n, vocab] of every position (and the residual stream after every layer)."""
    eps = cfg["norm"]["eps"]
    x = w["embed"][torch.as_tensor(list(tokens), dtype=torch.long)]
    kept = []
    for l, layer in enumerate(cfg["layers"]):
        p = f"l{l}."
        x = x + rms_norm(MIXERS[layer["type"]](x, w, p + "mix.", layer["mixer"], eps), w[p + "norm1"], eps)
        if layer["mlp"] is not None:
            x = x + rms_norm(dense_ff(x, w, p + "mlp.", layer["mlp"]["limit"]), w[p + "norm2"], eps)
        kept.append(x)
    logits = linear(rms_norm(x, w["final.norm"], eps), w["embed"])
    return (logits, torch.stack(kept)) if keep_layers else logits


# ---- seeded small models -----------------------------------------------------------------------------------------------------
def tensor_shapes(cfg):
    """Name -> shape of every tensor of a model."""
    W = cfg["width"]
    s = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    for l, layer in enumerate(cfg["layers"]):
        p, m = f"l{l}.", layer["mixer"]
        H, d, e = m["heads"], m["dim"], m["vdim"]
        s[p + "norm1"] = (W,)
        s[p + "mix.q"] = (H * d, W)
        s[p + "mix.o"] = (W, H * e)
        if layer["type"] == "attention":
            s.update({p + "mix.k": (m["kv_heads"] * d, W), p + "mix.q.norm": (d,), p + "mix.k.norm": (d,), p + "mix.g": (H, W)})
        else:
            s.update({p + "mix.k": (H * d, W), p + "mix.v": (H * e, W), p + "mix.g": (H * e, W), p + "mix.norm": (H * e,),
                      p + "mix.i": (H, W), p + "mix.i.b": (H,), p + "mix.f": (H, W), p + "mix.f.b": (H,)})
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            s.update({p + "norm2": (W,), p + "mlp.gate": (F, W), p + "mlp.up": (F, W), p + "mlp.down": (W, F)})
    return s


def random_weights(cfg, seed=0, scale=1.0):
    """bfloat16-representable random weights (float32 tensors)."""
    g = torch.Generator().manual_seed(seed)
    w = {}
    for name, shape in tensor_shapes(cfg).items():
        t = torch.randn(shape, generator=g)
        if name == "embed":
            t = t * 1.0
        elif "norm" in name.rsplit(".", 1)[-1]:
            t = 1.0 + 0.2 * t
        elif name.endswith(".i.b"):
            t = 0.5 * t - 1.0
        elif name.endswith(".f.b"):
            t = 2.0 + 1.5 * t                      # from strong forgetting to almost none
        elif name.endswith((".i", ".f")):
            t = t * 0.5 * scale * shape[-1] ** -0.5
        else:
            t = t * scale * shape[-1] ** -0.5
        w[name] = t.bfloat16().float()
    return w
