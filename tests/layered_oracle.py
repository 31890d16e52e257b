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


# ---- recurrences with a decay and no normaliser ----------------------------------------------------------------------------------
def silu(x):
    return x * torch.sigmoid(x)


def rotate_half(x, first_position, base, dims):
    """x [n, heads, d]: dimension i pairs with i + dims / 2; dimensions from ``dims`` on pass."""
    n, half = x.shape[0], dims // 2
    pos = torch.arange(first_position, first_position + n, dtype=x.dtype)
    freq = torch.tensor([base ** (-2.0 * i / dims) for i in range(half)], dtype=x.dtype)
    a = pos[:, None] * freq[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., :half], x[..., half:dims]
    return torch.cat([u * c - v * s, v * c + u * s, x[..., dims:]], dim=-1)


def decayed_memory(q, k, v, a, b, state=None):
    """One head, token by token: S <- a_t S + b_t k_t v_t^T, o_t = S^T q_t.  q, k [n, d], v [n, e], a, b [n].  Returns (o, S)."""
    S = torch.zeros(q.shape[1], v.shape[1], dtype=q.dtype) if state is None else state
    out = []
    for t in range(q.shape[0]):
        S = a[t] * S + b[t] * torch.outer(k[t], v[t])
        out.append(S.T @ q[t])
    return torch.stack(out), S


def fixed_decay_heads(q, k, v, decay):
    """q, k [n, H, d], v [n, H, e] -> o [n, H, e]."""
    one = torch.ones(q.shape[0], dtype=q.dtype)
    return torch.stack([decayed_memory(q[:, h], k[:, h], v[:, h], decay[h] * one, one)[0] for h in range(q.shape[1])], dim=1)


def retention_mixer(h, w, p, m, eps):
    n, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    rot = lambda x: rotate_half(x.view(n, H, d), 0, m["rot"]["base"], m["rot"]["dims"])
    q, k = rot(linear(h, w[p + "q"])), rot(linear(h, w[p + "k"])) * d ** -0.5
    o = fixed_decay_heads(q, k, linear(h, w[p + "v"]).view(n, H, e), m["decay"])
    return linear(rms(o, eps).reshape(n, H * e) * silu(linear(h, w[p + "g"])), w[p + "o"])


def lightning_mixer(h, w, p, m, eps):
    n, H, d, e = h.shape[0], m["heads"], m["dim"], m["vdim"]
    q, k, v = (silu(linear(h, w[p + c])) for c in "qkv")
    o = fixed_decay_heads(q.view(n, H, d), k.view(n, H, d), v.view(n, H, e), m["decay"]).reshape(n, H * e)
    return linear(rms_norm(o, w[p + "norm"], eps) * torch.sigmoid(linear(h, w[p + "g"])), w[p + "o"])


def causal_conv(x, weight, bias):
    """x [n, C], weight [C, taps]: the last column is the current token's; zeros before the start."""
    taps = weight.shape[1]
    out = bias.expand_as(x).clone()
    for j in range(taps):
        back = taps - 1 - j
        if back < x.shape[0]:
            out[back:] += x[: x.shape[0] - back] * weight[:, j]
    return out


def grouped_rms(x, parts, eps):
    return rms(x.reshape(x.shape[0], parts, -1), eps).reshape(x.shape)


def mamba2_mixer(h, w, p, m, eps):
    n, H, e, N, G = h.shape[0], m["heads"], m["vdim"], m["state"], m["groups"]
    inner = H * e
    z, xbc, dt = torch.split(linear(h, w[p + "in"]), [inner, inner + 2 * G * N, H], dim=-1)
    xbc = silu(causal_conv(xbc, w[p + "conv"], w[p + "conv.b"]))
    x, B, C = torch.split(xbc, [inner, G * N, G * N], dim=-1)
    x, B, C = x.reshape(n, H, e), B.reshape(n, G, N), C.reshape(n, G, N)
    dt = torch.nn.functional.softplus(dt + w[p + "dt_bias"])
    a = torch.exp(-torch.exp(w[p + "A_log"]) * dt)
    y = torch.stack([decayed_memory(C[:, i // (H // G)], B[:, i // (H // G)], x[:, i], a[:, i], dt[:, i])[0] + w[p + "D"][i] * x[:, i] for i in range(H)], dim=1)
    y = grouped_rms(y.reshape(n, inner) * silu(z), m["norm_groups"], eps) * w[p + "norm"]
    return linear(y, w[p + "o"])


# ---- softmax attention with normalised heads, a query temperature and capped scores -------------------------------------------------
def query_temperature(n, coef, every):
    return torch.tensor([1.0 + coef * math.log(math.floor((p + 1) / every) + 1) for p in range(n)], dtype=torch.float64)


def capped_attention(q, k, v, scale, softcap):
    """One head over all earlier positions."""
    n = q.shape[0]
    s = soft_cap((q @ k.T) * scale, softcap)
    return torch.softmax(s.masked_fill(torch.ones(n, n).triu(1).bool(), float("-inf")), dim=-1) @ v


def capped_attention_mixer(h, w, p, m, eps):
    n, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q, k = rms(linear(h, w[p + "q"]).view(n, H, d), eps), rms(linear(h, w[p + "k"]).view(n, G, d), eps)
    v = linear(h, w[p + "v"]).view(n, G, e)
    q = q * query_temperature(n, m["q_temp"]["coef"], m["q_temp"]["every"]).to(q.dtype)[:, None, None]
    o = torch.stack([capped_attention(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], m["scale"], m["softcap"]) for a in range(H)], dim=1)
    return linear(o.reshape(n, H * e), w[p + "o"])


def parallel_mixer(h, w, p, m, eps):
    return m["left_scale"] * capped_attention_mixer(h, w, p + "left.", m["left"], eps) + m["right_scale"] * mamba2_mixer(h, w, p + "right.", m["right"], eps)


def squared_relu_ff(x, w, p):
    return linear(torch.relu(linear(x, w[p + "up"])) ** 2, w[p + "down"])


# ---- interleaved rotation with scaled frequencies, attention with a sink, latent attention ----------------------------------------------
def frequencies(rot):
    """Angles per position of the ``dims`` / 2 pairs; long wavelengths are stretched by ``factor``, with a ramp in between."""
    out = []
    for i in range(rot["dims"] // 2):
        f = rot["base"] ** (-2.0 * i / rot["dims"])
        sc = rot.get("scaling")
        if sc is not None:
            turns = sc["original"] * f / (2.0 * math.pi)         # turns within the original context
            if turns < sc["low"]:
                f = f / sc["factor"]
            elif turns <= sc["high"]:
                s = (turns - sc["low"]) / (sc["high"] - sc["low"])
                f = (1.0 - s) * f / sc["factor"] + s * f
        out.append(f)
    return out


def rotate_pairs(x, first_position, rot):
    """x [n, heads, d]: dimensions 2i and 2i + 1 are a pair; dimensions from ``dims`` on pass."""
    dims = rot["dims"]
    pos = torch.arange(first_position, first_position + x.shape[0], dtype=x.dtype)
    a = pos[:, None] * torch.tensor(frequencies(rot), dtype=x.dtype)[None, :]
    c, s = torch.cos(a)[:, None, :], torch.sin(a)[:, None, :]
    u, v = x[..., 0:dims:2], x[..., 1:dims:2]
    out = x.clone()
    out[..., 0:dims:2] = u * c - v * s
    out[..., 1:dims:2] = v * c + u * s
    return out


def sink_attention(q, k, v, scale, sink=None):
    """One head over all earlier positions; the sink is one more term of the denominator (None: no sink)."""
    n = q.shape[0]
    s = ((q @ k.T) * scale).masked_fill(torch.ones(n, n).triu(1).bool(), float("-inf"))
    if sink is None:
        return torch.softmax(s, dim=-1) @ v
    return torch.softmax(torch.cat([s, sink.expand(n, 1)], dim=-1), dim=-1)[:, :n] @ v


def rotary_attention_mixer(h, w, p, m, shared):
    """Grouped-query attention with rotated heads and sinks; ``shared``: the keys and values of each layer so far."""
    n, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    q = rotate_pairs(linear(h, w[p + "q"]).view(n, H, d), 0, m["rot"])
    if "kv_from" in m:
        k, v = shared[m["kv_from"]]
    else:
        k = rotate_pairs(linear(h, w[p + "k"]).view(n, G, d), 0, m["rot"])
        v = linear(h, w[p + "v"]).view(n, G, e)
    o = torch.stack([sink_attention(q[:, a], k[:, a // (H // G)], v[:, a // (H // G)], m["scale"], w[p + "sink"][a]) for a in range(H)], dim=1)
    return linear(o.reshape(n, H * e), w[p + "o"]), (k, v)


def latent_attention_mixer(h, w, p, m, eps):
    """Keys and values are expanded from one normalised latent per token; one rotated key part serves all heads."""
    n, H, d, r, e, R = h.shape[0], m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    q = linear(h, w[p + "q"]).view(n, H, d + r)
    q = torch.cat([q[..., :d], rotate_pairs(q[..., d:], 0, m["rot"])], dim=-1)
    ckr = linear(h, w[p + "dkv"])
    c = rms_norm(ckr[:, :R], w[p + "dkv.norm"], eps)
    kr = rotate_pairs(ckr[:, None, R:], 0, m["rot"])
    k = torch.cat([linear(c, w[p + "uk"]).view(n, H, d), kr.expand(n, H, r)], dim=-1)
    v = linear(c, w[p + "uv"]).view(n, H, e)
    o = torch.stack([sink_attention(q[:, a], k[:, a], v[:, a], m["scale"]) for a in range(H)], dim=1).reshape(n, H * e)
    return linear(o * torch.sigmoid(linear(h, w[p + "g"])), w[p + "o"])


# ---- experts ---------------------------------------------------------------------------------------------------------------------
def route(z, correction, top, groups, keep, scale):
    """One token: chosen experts (best first) and their weights.  z [experts]: router logits."""
    s = torch.sigmoid(z)
    choice = s + correction
    size = len(choice) // groups
    best = sorted(range(groups), key=lambda g: -float(torch.sort(choice[g * size:(g + 1) * size], descending=True).values[:2].sum()))[:keep]
    allowed = [e for e in range(len(choice)) if e // size in best]
    chosen = sorted(allowed, key=lambda e: -float(choice[e]))[:top]
    weights = torch.stack([s[e] for e in chosen])
    return chosen, weights / (weights.sum() + 1e-20) * scale


def route_margin(z, correction, top, groups, keep):
    """How far the choice is from another one: the smaller of the gaps behind the last kept group and behind the last chosen expert."""
    choice = torch.sigmoid(z) + correction
    size = len(choice) // groups
    sums = torch.stack([torch.sort(choice[g * size:(g + 1) * size], descending=True).values[:2].sum() for g in range(groups)])
    order = torch.argsort(sums, descending=True)
    gap = float(sums[order[keep - 1]] - sums[order[keep]]) if keep < groups else math.inf
    left = torch.sort(torch.cat([choice[g * size:(g + 1) * size] for g in order[:keep].tolist()]), descending=True).values
    return min(gap, float(left[top - 1] - left[top])) if top < len(left) else gap


def expert(x, w, p):
    return linear(silu(linear(x, w[p + "gate"])) * linear(x, w[p + "up"]), w[p + "down"])


def experts_ff(h, w, p, mlp):
    r, out = mlp["router"], []
    z = linear(h, w[p + "router"])
    for t in range(h.shape[0]):
        chosen, weights = route(z[t], w[p + "correction"], r["top"], r["groups"]["count"], r["groups"]["keep"], r["scale"])
        out.append(sum(g * expert(h[t], w, f"{p}e{e}.") for e, g in zip(chosen, weights)))
    return torch.stack(out)


def layer_norm(x, weight, eps):
    d = x - x.mean(-1, keepdim=True)
    return d / torch.sqrt((d * d).mean(-1, keepdim=True) + eps) * weight


# ---- differential attention in chunks, element-wise recurrences, experts with a shared one, loops ----------------------------------------
def chunk_mask(n, size):
    """Position i sees j <= i of its own chunk of ``size`` positions."""
    i, j = torch.arange(n)[:, None], torch.arange(n)[None, :]
    return (j <= i) & (i // size == j // size)


def masked_attention(q, k, v, scale, mask):
    """One head (one map): q, k [n, d], v [n, e]."""
    return torch.softmax(((q @ k.T) * scale).masked_fill(~mask, float("-inf")), dim=-1) @ v


def difference_factor(w, p, diff):
    return torch.exp((w[p + "lq1"] * w[p + "lk1"]).sum()) - torch.exp((w[p + "lq2"] * w[p + "lk2"]).sum()) + diff


def differential_mixer(h, w, p, m, eps):
    """Two softmax maps per head over the same values; the second is taken off, the difference normalised per head, then gated."""
    n, H, G, d, e = h.shape[0], m["heads"], m["kv_heads"], m["dim"], m["vdim"]
    project = lambda c: linear(h, w[p + c]) + w[p + c + ".b"]
    q = rms_norm(project("q").view(n, 2 * H, d), w[p + "q.norm"], eps)
    k = rms_norm(project("k").view(n, 2 * G, d), w[p + "k.norm"], eps)
    q, k = (rotate_pairs(x, 0, m["rot"]) if m["rot"]["dims"] else x for x in (q, k))
    v = project("v").view(n, G, e)
    mask, lam = chunk_mask(n, m["mask"]["size"]), difference_factor(w, p, m["diff"])
    out = []
    for a in range(H):
        g = a // (H // G)
        a1, a2 = (masked_attention(q[:, 2 * a + i], k[:, 2 * g + i], v[:, g], m["scale"], mask) for i in (0, 1))
        out.append(rms(a1 - lam * a2, eps) * (1.0 - m["diff"]))
    o = torch.stack(out, dim=1).reshape(n, H * e) * torch.sigmoid(linear(h, w[p + "g"]))
    return linear(o, w[p + "o"]) + w[p + "o.b"]


def mingru_candidate(u):
    return torch.where(u >= 0, u + 0.5, torch.sigmoid(u))


def mingru_scan(z, c, state=None):
    """S <- (1 - z) S + z c for z, c [n, width]; every state, [n, width]."""
    S, out = torch.zeros(z.shape[1], dtype=z.dtype) if state is None else state, []
    for t in range(z.shape[0]):
        S = (1.0 - z[t]) * S + z[t] * c[t]
        out.append(S)
    return torch.stack(out)


def mingru_mixer(h, w, p, m, eps):
    z = torch.sigmoid(linear(h, w[p + "z"]) + w[p + "z.b"])
    S = mingru_scan(z, mingru_candidate(linear(h, w[p + "x"]) + w[p + "x.b"]))
    return linear(S * silu(linear(h, w[p + "g"])), w[p + "o"])


def selective_scan(x, dt, A, B, C, D, state=None):
    """x, dt [n, channels], A [channels, N], B, C [n, N], D [channels]: y [n, channels] and the last state."""
    S, out = torch.zeros_like(A) if state is None else state, []
    for t in range(x.shape[0]):
        S = torch.exp(dt[t][:, None] * A) * S + (dt[t] * x[t])[:, None] * B[t][None, :]
        out.append(S @ C[t] + D * x[t])
    return torch.stack(out), S


def mamba1_mixer(h, w, p, m, eps):
    inner, R, N = m["inner"], m["dt_rank"], m["state"]
    x, z = torch.split(linear(h, w[p + "in"]), [inner, inner], dim=-1)
    x = silu(causal_conv(x, w[p + "conv"], w[p + "conv.b"]))
    dt, B, C = torch.split(linear(x, w[p + "x"]), [R, N, N], dim=-1)
    dt = torch.nn.functional.softplus(linear(dt, w[p + "dt"]) + w[p + "dt.b"])
    y, _ = selective_scan(x, dt, -torch.exp(w[p + "A_log"]), B, C, w[p + "D"])
    return linear(y * silu(z), w[p + "o"])


def gelu_tanh(z):
    return 0.5 * z * (1.0 + torch.tanh(math.sqrt(2.0 / math.pi) * (z + 0.044715 * z ** 3)))


def gelu_ff(h, w, p):
    return linear(gelu_tanh(linear(h, w[p + "gate"])) * linear(h, w[p + "up"]), w[p + "down"])


def softmax_route(z, top):
    """One token: the experts with the largest scores (best first) and these scores."""
    s = torch.softmax(z, dim=-1)
    chosen = sorted(range(len(s)), key=lambda e: -float(s[e]))[:top]
    return chosen, torch.stack([s[e] for e in chosen])


def shared_experts_ff(h, w, p, mlp):
    """Chosen experts, weighted by their softmax scores, and one expert for every token behind a sigmoid."""
    z, limit, out = linear(h, w[p + "router"]), mlp["expert"]["limit"], []
    for t in range(h.shape[0]):
        chosen, weights = softmax_route(z[t], mlp["router"]["top"])
        out.append(sum(g * dense_ff(h[t], w, f"{p}e{e}.", limit) for e, g in zip(chosen, weights)))
    out = torch.stack(out)
    if mlp.get("shared") is not None:
        out = out + torch.sigmoid(linear(h, w[p + "shared.sg"])) * dense_ff(h, w, p + "shared.", mlp["shared"]["limit"])
    return out


def grouped_norm(x, weight, groups, eps):
    return grouped_rms(x, groups, eps) * weight


def plus_conv(h, weight):
    return h + causal_conv(h, weight, torch.zeros(h.shape[1], dtype=h.dtype))


def naforax_layer(x, w, p, layer, norm, mult):
    mixer = {"attention": differential_mixer, "mingru": mingru_mixer, "mamba1": mamba1_mixer}[layer["type"]]
    groups, eps = norm["groups"], norm["eps"]
    h = plus_conv(grouped_norm(x, w[p + "norm1"], groups, eps), w[p + "canon1"])
    x = x + mult * grouped_norm(mixer(h, w, p + "mix.", layer["mixer"], eps), w[p + "norm1b"], groups, eps)
    if layer["mlp"] is not None:
        h = plus_conv(grouped_norm(x, w[p + "norm2"], groups, eps), w[p + "canon2"])
        y = gelu_ff(h, w, p + "mlp.") if layer["mlp"]["kind"] == "dense" else shared_experts_ff(h, w, p + "mlp.", layer["mlp"])
        x = x + mult * grouped_norm(y, w[p + "norm2b"], groups, eps)
    return x


def loop_runs(layers, loop):
    """(layer, pass; None outside the loop) in the order they run."""
    start, stop, times = loop["start"], loop["stop"], loop["times"]
    return [(i, None) for i in range(start)] + [(i, t) for t in range(times) for i in range(start, stop)] + [(i, None) for i in range(stop, layers)]


def naforax_forward(cfg, w, tokens, keep_layers=False):
    first = w["embed"][torch.as_tensor(list(tokens), dtype=torch.long)]
    x, kept, norm, cap = first, [], cfg["norm"], cfg["logit_softcap"]
    for i, t in loop_runs(len(cfg["layers"]), cfg["loop"]):
        if t is not None and i == cfg["loop"]["start"]:
            x = x + w["loop.step"][t] + (first if t > 0 else 0.0)
        x = naforax_layer(x, w, f"l{i}.", cfg["layers"][i], norm, cfg["residual_mult"])
        kept.append(x)
    logits = soft_cap(linear(grouped_norm(x, w["final.norm"], norm["groups"], norm["eps"]), w["head"]), cap)
    return (logits, torch.stack(kept)) if keep_layers else logits


# ---- whole models -----------------------------------------------------------------------------------------------------------------
MIXERS = {"attention": attention_mixer, "mlstm": mlstm_mixer, "retention": retention_mixer, "lightning": lightning_mixer, "parallel": parallel_mixer}


def keripel_layer(x, w, p, layer, eps):
    """Norms on the sublayers' outputs only."""
    x = x + rms_norm(MIXERS[layer["type"]](x, w, p + "mix.", layer["mixer"], eps), w[p + "norm1"], eps)
    if layer["mlp"] is not None:
        x = x + rms_norm(dense_ff(x, w, p + "mlp.", layer["mlp"]["limit"]), w[p + "norm2"], eps)
    return x


def kekevik_layer(x, w, p, layer, eps):
    """A norm before and a norm after each sublayer."""
    y = MIXERS[layer["type"]](rms_norm(x, w[p + "norm1"], eps), w, p + "mix.", layer["mixer"], eps)
    x = x + rms_norm(y, w[p + "norm1b"], eps)
    if layer["mlp"] is not None:
        x = x + rms_norm(squared_relu_ff(rms_norm(x, w[p + "norm2"], eps), w, p + "mlp."), w[p + "norm2b"], eps)
    return x


def kutepel_layer(x, w, p, layer, eps, mult, shared):
    """One layer norm, the mixer and the feed-forward side by side behind it.  Returns x and the layer's keys and values."""
    h, m, kv = layer_norm(x, w[p + "norm1"], eps), layer["mixer"], None
    if layer["type"] == "attention":
        y, kv = rotary_attention_mixer(h, w, p + "mix.", m, shared)
    else:
        y = latent_attention_mixer(h, w, p + "mix.", m, eps)
    if layer["mlp"] is not None:
        y = y + experts_ff(h, w, p + "mlp.", layer["mlp"])
    return x + mult * y, kv


def forward(cfg, w, tokens, keep_layers=False):
    """Logits [n, vocab] of every position (and the residual stream after every layer)."""
    eps, arch = cfg["norm"]["eps"], cfg["architecture"]
    if arch == "Naforax":
        return naforax_forward(cfg, w, tokens, keep_layers)
    x = w["embed"][torch.as_tensor(list(tokens), dtype=torch.long)] * cfg.get("embedding", {}).get("scale", 1.0)
    kept, shared = [], []
    for l, layer in enumerate(cfg["layers"]):
        if arch == "Kutepel":
            x, kv = kutepel_layer(x, w, f"l{l}.", layer, eps, cfg["residual_mult"], shared)
            shared.append(kv)
        else:
            x = {"Keripel": keripel_layer, "Kekevik": kekevik_layer}[arch](x, w, f"l{l}.", layer, eps)
        kept.append(x)
    norm = layer_norm if arch == "Kutepel" else rms_norm
    logits = linear(norm(x, w["final.norm"], eps), w["embed"])
    return (logits, torch.stack(kept)) if keep_layers else logits


# ---- seeded small models -----------------------------------------------------------------------------------------------------
def keripel_mixer_shapes(layer, p, W):
    m = layer["mixer"]
    H, d, e = m["heads"], m["dim"], m["vdim"]
    s = {p + "q": (H * d, W), p + "o": (W, H * e)}
    if layer["type"] == "attention":
        s.update({p + "k": (m["kv_heads"] * d, W), p + "q.norm": (d,), p + "k.norm": (d,), p + "g": (H, W)})
    else:
        s.update({p + "k": (H * d, W), p + "v": (H * e, W), p + "g": (H * e, W), p + "norm": (H * e,),
                  p + "i": (H, W), p + "i.b": (H,), p + "f": (H, W), p + "f.b": (H,)})
    return s


def kekevik_mixer_shapes(layer, p, W):
    m = layer["mixer"]
    if layer["type"] == "parallel":
        a, b = m["left"], m["right"]
        G, inner = a["kv_heads"], b["heads"] * b["vdim"]
        C = inner + 2 * b["groups"] * b["state"]
        l, r = p + "left.", p + "right."
        return {l + "q": (a["heads"] * a["dim"], W), l + "k": (G * a["dim"], W), l + "v": (G * a["vdim"], W), l + "o": (W, a["heads"] * a["vdim"]),
                r + "in": (inner + C + b["heads"], W), r + "conv": (C, b["conv"]), r + "conv.b": (C,), r + "dt_bias": (b["heads"],),
                r + "A_log": (b["heads"],), r + "D": (b["heads"],), r + "norm": (inner,), r + "o": (W, inner)}
    H, d, e = m["heads"], m["dim"], m["vdim"]
    s = {p + "q": (H * d, W), p + "k": (H * d, W), p + "v": (H * e, W), p + "g": (H * e, W), p + "o": (W, H * e)}
    if layer["type"] == "lightning":
        s[p + "norm"] = (H * e,)
    return s


def kutepel_tensor_shapes(cfg):
    W = cfg["width"]
    s = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    for l, layer in enumerate(cfg["layers"]):
        m, p, f = layer["mixer"], f"l{l}.mix.", f"l{l}.mlp."
        H, d, e = m["heads"], m["dim"], m["vdim"]
        s[f"l{l}.norm1"] = (W,)
        if layer["type"] == "attention":
            s.update({p + "q": (H * d, W), p + "sink": (H,)})
            if "kv_from" not in m:
                s.update({p + "k": (m["kv_heads"] * d, W), p + "v": (m["kv_heads"] * e, W)})
        else:
            R, r = m["kv_rank"], m["rot_dim"]
            s.update({p + "q": (H * (d + r), W), p + "dkv": (R + r, W), p + "dkv.norm": (R,), p + "uk": (H * d, R), p + "uv": (H * e, R), p + "g": (H * e, W)})
        s[p + "o"] = (W, H * e)
        if layer["mlp"] is not None:
            E, F = layer["mlp"]["router"]["experts"], layer["mlp"]["expert"]["ff"]
            s.update({f + "router": (E, W), f + "correction": (E,)})
            for j in range(E):
                s.update({f"{f}e{j}.gate": (F, W), f"{f}e{j}.up": (F, W), f"{f}e{j}.down": (W, F)})
    return s


def naforax_tensor_shapes(cfg):
    W, V, taps = cfg["width"], cfg["vocab"], cfg["canon"]["taps"]
    s = {"embed": (V, W), "head": (V, W), "final.norm": (W,), "loop.step": (cfg["loop"]["times"], W)}
    for l, layer in enumerate(cfg["layers"]):
        m, p, f, mlp = layer["mixer"], f"l{l}.mix.", f"l{l}.mlp.", layer["mlp"]
        for n in ("1", "2") if mlp is not None else ("1",):
            s.update({f"l{l}.norm{n}": (W,), f"l{l}.norm{n}b": (W,), f"l{l}.canon{n}": (W, taps)})
        if layer["type"] == "attention":
            H, G, d, e = m["heads"], m["kv_heads"], m["dim"], m["vdim"]
            for n, rows in (("q", 2 * H * d), ("k", 2 * G * d), ("v", G * e)):
                s.update({p + n: (rows, W), p + n + ".b": (rows,)})
            s.update({p + n: (d,) for n in ("q.norm", "k.norm", "lq1", "lk1", "lq2", "lk2")})
            s.update({p + "g": (H * e, W), p + "o": (W, H * e), p + "o.b": (W,)})
        elif layer["type"] == "mingru":
            E = m["width"]
            s.update({p + "z": (E, W), p + "z.b": (E,), p + "x": (E, W), p + "x.b": (E,), p + "g": (E, W), p + "o": (W, E)})
        else:
            C, N, R = m["inner"], m["state"], m["dt_rank"]
            s.update({p + "in": (2 * C, W), p + "conv": (C, m["conv"]), p + "conv.b": (C,), p + "x": (R + 2 * N, C), p + "dt": (C, R), p + "dt.b": (C,),
                      p + "A_log": (C, N), p + "D": (C,), p + "o": (W, C)})
        block = lambda q, F: {q + "gate": (F, W), q + "up": (F, W), q + "down": (W, F)}
        if mlp is not None and mlp["kind"] == "dense":
            s.update(block(f, mlp["ff"]))
        elif mlp is not None:
            s[f + "router"] = (mlp["router"]["experts"], W)
            for j in range(mlp["router"]["experts"]):
                s.update(block(f"{f}e{j}.", mlp["expert"]["ff"]))
            if mlp.get("shared") is not None:
                s.update({**block(f + "shared.", mlp["shared"]["ff"]), f + "shared.sg": (1, W)})
    return s


def tensor_shapes(cfg):
    """Name -> shape of every tensor of a model."""
    if cfg["architecture"] == "Naforax":
        return naforax_tensor_shapes(cfg)
    if cfg["architecture"] == "Kutepel":
        return kutepel_tensor_shapes(cfg)
    W, keripel = cfg["width"], cfg["architecture"] == "Keripel"
    s = {"embed": (cfg["vocab"], W), "final.norm": (W,)}
    for l, layer in enumerate(cfg["layers"]):
        p, tail = f"l{l}.", [""] if keripel else ["", "b"]
        s.update({p + "norm1" + t: (W,) for t in tail})
        s.update((keripel_mixer_shapes if keripel else kekevik_mixer_shapes)(layer, p + "mix.", W))
        if layer["mlp"] is not None:
            F = layer["mlp"]["ff"]
            s.update({p + "norm2" + t: (W,) for t in tail})
            s.update({p + "mlp." + n: (F, W) for n in (["gate", "up"] if keripel else ["up"])})
            s[p + "mlp.down"] = (W, F)
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
        elif name.endswith("dt_bias"):
            t = t - 1.0
        elif name.endswith(".sink"):
            t = 1.0 + t
        elif name.endswith(".correction"):
            t = 0.3 * t - 0.2                      # some choice scores are negative
        elif name.endswith(".dt.b"):
            t = t - 2.0                            # step sizes around an eighth
        elif name.endswith((".q.b", ".k.b", ".v.b", ".o.b", ".z.b", ".x.b")):
            t = 0.4 * t
        elif name.endswith((".lq1", ".lk1", ".lq2", ".lk2")):
            t = 1.2 * t * shape[0] ** -0.5
        elif ".canon" in name:
            t = 0.35 * t
        elif name == "loop.step":
            t = 0.3 * t
        elif name.endswith("A_log"):
            t = 1.5 * t - 2.0                      # from forgetting in a few tokens to hardly at all
        elif name.endswith(".D"):
            t = 1.0 + 0.3 * t
        elif name.endswith("conv.b"):
            t = 0.2 * t
        elif name.endswith((".i", ".f")):
            t = t * 0.5 * scale * shape[-1] ** -0.5
        else:
            t = t * scale * shape[-1] ** -0.5
        w[name] = t.bfloat16().float()
    if cfg["architecture"] == "Kutepel":
        settle_routers(cfg, w, g)
    elif cfg["architecture"] == "Naforax":
        settle_softmax_routers(cfg, w, g)
    return w


CODES = 16


def settle_routers(cfg, w, g, margin=0.016):
    """Makes the choice of experts depend on the token alone, clearly: the last ``CODES`` dimensions of the stream hold a code of the token
    that no sublayer changes, and router rows read only those.  The last code balances the rows, so that a mean does not enter."""
    W, amp = cfg["width"], 6.0
    code = torch.randint(0, CODES - 1, (cfg["vocab"],), generator=g)
    w["embed"][:, -CODES:] = amp * torch.nn.functional.one_hot(code, CODES).float()
    for l, layer in enumerate(cfg["layers"]):
        p = f"l{l}."
        w[p + "norm1"][-CODES:] = 1.0
        w[p + "mix.o"][-CODES:] = 0.0
        if layer["mlp"] is None:
            continue
        r, c = layer["mlp"]["router"], w[p + "mlp.correction"]
        E, groups, keep = r["experts"], r["groups"]["count"], r["groups"]["keep"]
        for e in range(E):
            w[f"{p}mlp.e{e}.down"][-CODES:] = 0.0
        rows = torch.zeros(E, W)
        for i in range(CODES - 1):
            for _ in range(400):
                col = (torch.linspace(-0.7, 0.7, E)[torch.randperm(E, generator=g)] if E > 1 else torch.ones(1)).bfloat16().float()
                if all(route_margin(col * amp / f, c, r["top"], groups, keep) > margin for f in torch.linspace(0.88, 1.6, 25).tolist()):
                    break
            rows[:, W - CODES + i] = col
        rows[:, -1] = -rows.sum(1)
        w[p + "mlp.router"] = rows.bfloat16().float()


def settle_softmax_routers(cfg, w, g):
    """The same for routers that compare logits behind a norm without a mean, in a stream that a loop adds the embedding to: sublayers,
    convolutions and the loop's steps leave the code's dimensions alone, so that router logits are a positive multiple of well-spread ones."""
    layers = [l for l, layer in enumerate(cfg["layers"]) if layer["mlp"] is not None and layer["mlp"]["kind"] == "moe"]
    if not layers:
        return
    W = cfg["width"]
    code = torch.randint(0, CODES, (cfg["vocab"],), generator=g)
    w["embed"][:, -CODES:] = 6.0 * torch.nn.functional.one_hot(code, CODES).float()
    w["loop.step"][:, -CODES:] = 0.0
    for l, layer in enumerate(cfg["layers"]):
        p = f"l{l}."
        for n in ("1", "2") if layer["mlp"] is not None else ("1",):
            w[p + f"norm{n}"][-CODES:] = 1.0
            w[p + f"norm{n}b"][-CODES:] = 0.0
            w[p + f"canon{n}"][-CODES:] = 0.0
    for l in layers:
        E = cfg["layers"][l]["mlp"]["router"]["experts"]
        rows = torch.zeros(E, W)
        for i in range(CODES):
            rows[:, W - CODES + i] = torch.linspace(-0.6, 0.6, E)[torch.randperm(E, generator=g)] if E > 1 else torch.ones(1)
        w[f"l{l}.mlp.router"] = rows.bfloat16().float()
