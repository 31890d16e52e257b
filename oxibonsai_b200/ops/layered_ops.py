"""Torch-facing wrappers of the layer-list decoder kernels in ``libbonsai_layered.so`` (csrc/layered, the sampler and the
tcgen05 GEMM).  Every function launches on torch's current stream; there is no PyTorch fallback."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass

import torch

from .. import _native
from . import cuda_ops as K

_vp, _i, _f = C.c_void_p, C.c_int, C.c_float
_SIG = {
    "bonsai_lay_embed": [_vp, _i, _vp, _f, _i, _i, _vp, _vp, _i, _i, _vp, _f, _i, _vp],
    "bonsai_lay_norm_add": [_vp, _vp, _i, _vp, _f, _i, _i, _vp, _i, _i, _vp, _vp],
    "bonsai_lay_side_by_side": [_vp, _vp, _i, _vp, _i, _i, _vp, _i, _vp, _i, _f, _i, _i, _vp, _i, _i, _vp, _f, _i, _vp],
    "bonsai_lay_norm_rows": [_vp, _vp, _vp, _f, _i, _i, _i, _vp, _i, _i, _vp],
    "bonsai_lay_gated_norm": [_vp, _i, _vp, _i, _vp, _f, _i, _i, _i, _i, _i, _f, _vp, _i, _i, _vp],
    "bonsai_lay_linear_few": [_vp, _i, _i, _vp, _i, _i, _vp, _vp, _i, _i, _f, _f, _f, _f, _vp],
    "bonsai_lay_linear_f32": [_vp, _i, _i, _i, _vp, _i, _i, _vp, _i, _i, _f, _f, _f, _f, _vp],
    "bonsai_dense_gemm_bf16": [_vp, _i, _i, _vp, _i, _i, _vp, _vp, _i, _i, _f, _f, _f, _f, _vp, _vp, C.c_size_t, _i, _vp],
    "bonsai_bitgemm_prefill_ws_bytes": [],
    "bonsai_lay_attn_row": [_i],
    "bonsai_lay_attn_append": [_vp, _vp, _vp, _i, _i, _i, _vp],
    "bonsai_lay_attn_prompt": [_vp, _vp, _vp, _vp, _vp, _i, _vp],
    "bonsai_lay_attn_decode": [_vp, _vp, _vp, _i, _i, _vp],
    "bonsai_lay_attn_f32": [_vp, _vp, _vp, _i, _vp],
    "bonsai_lay_latent_row": [_i, _i],
    "bonsai_lay_latent_max_splits": [],
    "bonsai_lay_latent_max_cluster": [],
    "bonsai_lay_latent_group": [_i],
    "bonsai_lay_latent_append": [_vp, _vp, _vp, _i, _i, _i, _vp],
    "bonsai_lay_latent_query": [_vp, _vp, _vp, _i, _vp],
    "bonsai_lay_latent_decode": [_vp, _vp, _vp, _i, _i, _i, _vp],
    "bonsai_lay_latent_value": [_vp, _vp, _vp, _i, _i, _vp],
    "bonsai_lay_latent_gather": [_vp, _vp, _vp, _vp, _i, _i, _vp, _i, _vp],
    "bonsai_lay_latent_prompt": [_vp, _vp, _vp, _vp, _vp, _vp, _i, _vp, _i, _vp, _i, _vp],
    "bonsai_lay_latent_f32": [_vp, _vp, _vp, _i, _vp],
    "bonsai_lay_route_small": [_i],
    "bonsai_lay_route": [_vp, _vp, _vp, _i, _vp, _i, _i, _vp, _i, _vp],
    "bonsai_lay_experts_few": [_vp, _i, _i, _i, _vp, _i, _vp, _vp, _vp, _i, _i, _i, _vp, _i, _i, _f, _f, _f, _f, _vp],
    "bonsai_lay_experts_f32": [_vp, _i, _i, _i, _i, _vp, _i, _vp, _vp, _vp, _i, _i, _vp, _i, _i, _f, _f, _f, _f, _vp],
    "bonsai_grouped_gemm_bf16": [_vp, _i, _i, _i, _vp, _i, _i, _vp, _vp, _vp, _i, _i, _f, _f, _f, _f, _i, _vp, _i, _vp],
    "bonsai_lay_mlstm_dim": [_i],
    "bonsai_lay_mlstm_vdim": [_i],
    "bonsai_lay_mlstm_chunk_dim": [],
    "bonsai_lay_mlstm_fused_vdim": [],
    "bonsai_lay_mlstm_step": [_vp, _vp, _vp, _vp, _i, _i, _vp],
    "bonsai_lay_mlstm_chunk_tokens": [],
    "bonsai_lay_mlstm_chunk": [_vp, _vp, _vp, _vp, _i, _vp, _i, _vp, _vp],
    "bonsai_lay_rec_dim": [_i],
    "bonsai_lay_rec_vdim": [_i],
    "bonsai_lay_rec_features_width": [_i, _i, _i, _i],
    "bonsai_lay_rec_chunk_dim": [],
    "bonsai_lay_rec_fused_vdim": [],
    "bonsai_lay_rec_features": [_vp, _vp, _vp, _i, _i, _i, _vp],
    "bonsai_lay_rec_ring": [_vp, _vp, _vp, _vp, _i, _vp],
    "bonsai_lay_rec_step": [_vp, _vp, _vp, _vp, _i, _i, _i, _i, _vp],
    "bonsai_lay_rec_chunk": [_vp, _vp, _vp, _vp, _i, _vp, _i, _vp, _vp],
    "bonsai_lay_row_step": [_vp, _vp, _vp, _i, _vp, _i, _i, _vp, _i, _vp, _i, _vp, _i, _vp],
    "bonsai_lay_conv": [_vp, _vp, _vp, _i, _vp, _vp, _i, _vp],
    "bonsai_lay_conv_rows": [],
    "bonsai_lay_conv_taps": [],
    "bonsai_lay_gru_step": [_vp, _vp, _vp, _i, _i, _vp],
    "bonsai_lay_gru_scan": [_vp, _vp, _vp, _vp, _i, _i, _i, _vp],
    "bonsai_lay_gru_tokens": [],
    "bonsai_lay_scan_states": [_i],
    "bonsai_lay_scan_channels": [_i],
    "bonsai_lay_scan_step": [_vp, _vp, _vp, _i, _i, _vp],
    "bonsai_lay_scan": [_vp, _vp, _vp, _vp, _i, _vp, _i, _vp, _i, _vp],
    "bonsai_lay_narrow": [_vp, _i, _i, _i, _i, _vp, _i, _vp],
    "bonsai_sample": K._SIG["bonsai_sample"],
}
_lib = None
FEW_ROWS = 32               # rows up to which a projection goes to the weight-streaming kernel
FEW_MORE = (64, 2368)       # and that, where the matrix has at most so many outputs (16 per SM)
K_ALIGN = 128               # inputs of a bf16 projection are padded to a multiple of this


def lib() -> C.CDLL:
    global _lib
    if _lib is None:
        l = _native.layered()
        for name, args in _SIG.items():
            fn = getattr(l, name)
            fn.argtypes = args
            fn.restype = C.c_size_t if name.endswith("ws_bytes") else C.c_int
        _lib = l
    return _lib


def round_up(n: int, m: int) -> int:
    return -(-n // m) * m


class DenseWeight:
    """bf16 matrix [n, kp] on the device: ``k`` inputs, zero columns up to a multiple of 128.  ``columns[i]`` is the first
    output of part i; parts start at multiples of four outputs (zero rows in between)."""

    def __init__(self, parts: list[torch.Tensor], device, interleave: bool = False):
        self.k = parts[0].shape[1]
        assert all(p.shape[1] == self.k and p.dtype == torch.bfloat16 for p in parts)
        self.kp = round_up(self.k, K_ALIGN)
        if interleave:                       # rows 2j, 2j + 1 = row j of the two parts (the gated epilogue's order)
            a, b = parts
            self.columns, rows = [0, 1], [torch.stack([a, b], dim=1).reshape(-1, self.k)]
            self.n = 2 * a.shape[0]
        else:
            self.columns, rows, n = [], [], 0
            for p in parts:
                self.columns.append(n)
                pad = round_up(p.shape[0], 4) - p.shape[0] if len(parts) > 1 else 0
                rows += [p, torch.zeros((pad, self.k), dtype=torch.bfloat16)]
                n += p.shape[0] + pad
            self.n = n
        m = torch.zeros((self.n, self.kp), dtype=torch.bfloat16)
        m[:, : self.k] = torch.cat(rows)
        self.data = m.to(device)

    @property
    def nbytes(self) -> int:
        return self.data.numel() * 2


class GemmScratch:
    """Workspace and status word of the tcgen05 GEMM for one stream."""

    def __init__(self, device, status: torch.Tensor):
        self.ws = torch.zeros(int(lib().bonsai_bitgemm_prefill_ws_bytes()), dtype=torch.uint8, device=device)
        self.status = status
        self.sms = torch.cuda.get_device_properties(device).multi_processor_count


@dataclass(frozen=True)
class Glu:
    """Clamped gated unit over interleaved gate / up rows: g * sigmoid(alpha (g + cubic g^3)) * (u + offset)."""
    limit: float
    alpha: float
    offset: float
    cubic: float = 0.0

    @property
    def args(self) -> tuple[float, float, float, float]:
        return self.limit, self.alpha, self.offset, self.cubic


@dataclass(frozen=True)
class SoftCap:
    """f32 outputs become cap * tanh(output / cap)."""
    cap: float


SQUARED_RELU = "squared_relu"
_NO_GLU = Glu(0.0, 0.0, 0.0)


def linear(w: DenseWeight, x: torch.Tensor, T: int, out: torch.Tensor, scratch: GemmScratch, act: Glu | SoftCap | str | None = None) -> None:
    """out[:T] = act(x[:T] W^T).  bf16 ``x`` (row stride >= kp, finite in the padding): tensor cores, f32 or bf16 ``out`` (bf16 with
    a :class:`Glu` or ``SQUARED_RELU``, f32 with a :class:`SoftCap`); f32 ``x``: 32-bit throughout."""
    l, s = lib(), K.stream()
    if act is None:
        epi, glu = (3 if out.dtype == torch.bfloat16 else 0), _NO_GLU
    elif isinstance(act, SoftCap):
        epi, glu = 4, Glu(act.cap, 0.0, 0.0)
    else:
        epi, glu = (1, act) if isinstance(act, Glu) else (2, _NO_GLU)
    if x.dtype == torch.float32:
        K.check(l.bonsai_lay_linear_f32(w.data.data_ptr(), w.n, w.k, w.kp, x.data_ptr(), x.stride(0), T, out.data_ptr(), out.stride(0), epi, *glu.args, s),
                "linear_f32")
        return
    assert x.dtype == torch.bfloat16 and (out.dtype == torch.float32 if epi in (0, 4) else out.dtype == torch.bfloat16)
    f32, b16 = (out.data_ptr(), None) if epi in (0, 4) else (None, out.data_ptr())
    if T <= FEW_ROWS or (T <= FEW_MORE[0] and w.n <= FEW_MORE[1]):
        K.check(l.bonsai_lay_linear_few(w.data.data_ptr(), w.n, w.kp, x.data_ptr(), x.stride(0), T, f32, b16, out.stride(0), epi, *glu.args, s), "linear_few")
    else:
        K.check(l.bonsai_dense_gemm_bf16(w.data.data_ptr(), w.n, w.kp, x.data_ptr(), x.stride(0), T, f32, b16, out.stride(0), (0, 4, 5, 6, 7)[epi], *glu.args,
                                         scratch.status.data_ptr(), scratch.ws.data_ptr(), scratch.ws.numel(), scratch.sms, s), "dense_gemm_bf16")


def _row_out(t: torch.Tensor | None) -> tuple[int | None, int, int]:
    return (None, 0, 0) if t is None else (t.data_ptr(), t.stride(0), int(t.dtype == torch.float32))


def embed(table: torch.Tensor, tokens: torch.Tensor, scale: float, T: int, width: int, x: torch.Tensor, h: torch.Tensor | None,
          next_norm: torch.Tensor | None, eps: float, center: bool = False) -> None:
    """x = table[tokens] * scale; ``h`` receives x, or its norm with weight ``next_norm`` (``center``: a layer norm)."""
    K.check(lib().bonsai_lay_embed(table.data_ptr(), table.stride(0), tokens.data_ptr(), scale, T, width, x.data_ptr(), *_row_out(h), K.ptr(next_norm), eps,
                                   int(center), K.stream()), "embed")


def norm_add(x: torch.Tensor, y: torch.Tensor, w: torch.Tensor, eps: float, T: int, h: torch.Tensor | None, next_norm: torch.Tensor | None = None) -> None:
    """x += rmsnorm(y) * w over the first T rows; ``h`` receives x, or its norm with weight ``next_norm``."""
    K.check(lib().bonsai_lay_norm_add(x.data_ptr(), y.data_ptr(), y.stride(0), w.data_ptr(), eps, T, x.shape[1], *_row_out(h), K.ptr(next_norm), K.stream()),
            "norm_add")


def side_by_side(x: torch.Tensor, y: torch.Tensor, experts: "Routing | None", mult: float, T: int, h: torch.Tensor | None, next_norm: torch.Tensor | None,
                 eps: float, center: bool) -> None:
    """x += mult * (y + each row's expert outputs); ``h`` receives x, or its norm with weight ``next_norm``.  Leaves the router's
    counters zero."""
    e = (None, 0, 0, None, 0, None, 0) if experts is None else experts.outputs
    K.check(lib().bonsai_lay_side_by_side(x.data_ptr(), y.data_ptr(), y.stride(0), *e, mult, T, x.shape[1], *_row_out(h), K.ptr(next_norm), eps, int(center),
                                          K.stream()), "side_by_side")


class RowStep:
    """What happens between two sublayers, in one launch:
    ``x += mult * norm(sigmoid(gate) (y + bias) + expert rows) * w``, then ``x += scale * table[token] + step``, then ``n = norm(x) * next``
    and ``h = n + conv(n)``.  Every part may be left out; ``fresh``: x starts here.  ``rows``: positions, slots and tokens of the rows;
    ``conv``: weights [taps, width] (the current token's first) and the ring of earlier inputs.  Norms have ``groups`` parts."""

    def __init__(self, x: torch.Tensor, h: torch.Tensor | None, rows, state_table: torch.Tensor, *, eps: float, groups: int, mult: float = 1.0,
                 y: torch.Tensor | None = None, bias: torch.Tensor | None = None, gate: torch.Tensor | None = None, w: torch.Tensor | None = None,
                 table: torch.Tensor | None = None, scale: float = 1.0, step: torch.Tensor | None = None, next_norm: torch.Tensor | None = None,
                 conv: tuple[torch.Tensor, torch.Tensor] | None = None, n32: torch.Tensor | None = None, fresh: bool = False):
        ld = lambda t: 0 if t is None else t.stride(0)
        weight, ring = conv if conv is not None else (None, None)
        h_f32 = h is not None and h.dtype == torch.float32
        self.call = MixerCall([x, y, bias, gate, w, table, rows.tokens, step, next_norm, n32, h, weight, ring, rows.positions, rows.slots, state_table],
                              [ld(y), ld(gate), x.shape[1], groups, ld(table), ld(n32), ld(h), int(h_f32), 0 if weight is None else weight.shape[0], int(fresh)],
                              [eps, mult, scale])
        self.conv = None
        if conv is not None and n32 is not None:
            self.conv = Conv(n32, 0, x.shape[1], weight, None, ring, rows, state_table, h, add=True)

    def __call__(self, T: int, st, experts: "Routing | None" = None, norm_of: int | None = None) -> None:
        """``st``: the step's rows (single tokens and portions); ``norm_of``: device address of the rows whose norm alone is asked for."""
        e = (None, 0, 0, None, 0, None, 0) if experts is None else experts.outputs
        here = self.conv is None or not st.portions
        K.check(lib().bonsai_lay_row_step(*self.call.args, T, *e, norm_of, int(here), K.stream()), "row_step")
        if not here:
            self.conv(st)


class Conv:
    """Causal convolution over tokens, a row of ``channels`` columns per token: out = [x +] [silu] (conv(x) + bias)."""

    def __init__(self, x: torch.Tensor, col: int, channels: int, weight: torch.Tensor, bias: torch.Tensor | None, ring: torch.Tensor, rows,
                 state_table: torch.Tensor, out: torch.Tensor, add: bool = False, silu: bool = False):
        self.call = MixerCall([x, weight, bias, ring, rows.positions, rows.slots, state_table, out],
                              [x.stride(0), col, channels, weight.shape[0], out.stride(0), int(out.dtype == torch.float32), int(add), int(silu)], [])

    def __call__(self, st) -> None:
        tiles, n = st.tiles[lib().bonsai_lay_conv_rows()] if st.portions else (None, 0)
        K.check(lib().bonsai_lay_conv(*self.call.args, st.singles, st.entries if n else None, tiles, n, K.stream()), "conv")


def conv_weight(w: torch.Tensor) -> torch.Tensor:
    """[channels, taps] with the current token's tap last -> [taps, channels] with it first."""
    return w.flip(1).t().contiguous()


def narrow(x: torch.Tensor, col: int, n: int, T: int, out: torch.Tensor) -> None:
    """f32 columns ``col`` .. ``col + n - 1`` of the first T rows as bf16."""
    K.check(lib().bonsai_lay_narrow(x.data_ptr(), x.stride(0), col, n, T, out.data_ptr(), out.stride(0), K.stream()), "narrow")


def norm_rows(x: torch.Tensor, rows: int | None, count: int, w: torch.Tensor, eps: float, out: torch.Tensor, center: bool = False) -> None:
    """out[i] = rmsnorm(x[rows[i]]) * w (``rows``: device address of int32 indices, None = 0 .. count - 1); ``center``: a layer norm."""
    K.check(lib().bonsai_lay_norm_rows(x.data_ptr(), rows, w.data_ptr(), eps, int(center), count, x.shape[1], out.data_ptr(), out.stride(0),
                                       int(out.dtype == torch.float32), K.stream()), "norm_rows")


def gated_norm(o: torch.Tensor, row0: int, gate: torch.Tensor, gate_col: int, w: torch.Tensor | None, eps: float, T: int, parts: int, width: int,
               out: torch.Tensor, act: str = "sigmoid", gate_first: bool = False, scale: float = 1.0) -> None:
    """Rows row0 .. row0 + T - 1 of all three, in ``parts`` parts of ``width`` columns with their own root mean square:
    out = o / rms(o) * w * act(gate) * scale, or with ``gate_first`` the same of o * act(gate) without a gate behind."""
    K.check(lib().bonsai_lay_gated_norm(o.data_ptr() + 4 * row0 * o.stride(0), o.stride(0), gate.data_ptr() + 4 * (row0 * gate.stride(0) + gate_col),
                                        gate.stride(0), K.ptr(w), eps, T, parts, width, {"sigmoid": 0, "silu": 1}[act], int(gate_first), scale,
                                        out.data_ptr() + out.element_size() * row0 * out.stride(0), out.stride(0), int(out.dtype == torch.float32),
                                        K.stream()), "gated_norm")


class MixerCall:
    """The argument blocks (pointers, sizes, constants) of the launches of one mixer or step; the tensors must outlive it."""

    def __init__(self, ptrs: list[torch.Tensor | None], ints: list[int], floats: list[float]):
        self._keep = ptrs
        self.ptrs = (_vp * len(ptrs))(*[K.ptr(t) for t in ptrs])
        self.ints = (_i * len(ints))(*ints)
        self.floats = (_f * len(floats))(*floats)

    @property
    def args(self):
        return self.ptrs, self.ints, self.floats


class ExpertScratch:
    """Buffers the expert layers of a model share (they run one after another): the router's lists for ``rows`` tokens, and the sorted
    rows, hidden units and outputs of all (token, chosen expert) pairs."""

    def __init__(self, rows: int, width: int, specs, exact: bool, device):
        self.rows, self.width, self.exact = rows, width, exact
        top, experts = max(s.router.top for s in specs), max(s.router.experts for s in specs)
        self.pairs = rows * top
        i32, f32 = dict(dtype=torch.int32, device=device), dict(dtype=torch.float32, device=device)
        act = dict(dtype=torch.float32 if exact else torch.bfloat16, device=device)
        self.counts, self.lists = torch.zeros(experts, **i32), torch.zeros(2 * experts + 2, **i32)
        self.pair, self.pair_weight = torch.zeros((self.pairs, 2), **i32), torch.zeros(self.pairs, **f32)
        self.token, self.weight, self.at = torch.zeros(self.pairs, **i32), torch.zeros(self.pairs, **f32), torch.zeros(self.pairs, **i32)
        # the padding columns stay zero for the projections that read them: one buffer per number of hidden units
        self.sorted = None if exact else torch.zeros((self.pairs, round_up(width, K_ALIGN)), **act)
        self.hidden = {ff: torch.zeros((self.pairs, round_up(ff, 4 if exact else K_ALIGN)), **act) for ff in {s.ff for s in specs}}
        ld = round_up(width, 8)
        self.out = torch.zeros((self.pairs, ld), **act)
        # f32 outputs of steps with few pairs, in the same memory
        self.out32 = self.out if exact else self.out.view(-1).view(torch.float32)[: self.pairs // 2 * ld].view(-1, ld)


class Routing:
    """One expert layer's calls: choice, sorting, the experts' projections.  ``logits``: the projections the router's are part of."""

    def __init__(self, spec, up: DenseWeight, down: DenseWeight, correction: torch.Tensor | None, logits: torch.Tensor, column: int, scratch: ExpertScratch):
        r = spec.router
        self.spec, self.up, self.down, self.s = spec, up, down, scratch
        self.glu = Glu(spec.limit, spec.alpha, spec.offset)
        self.call = MixerCall([logits, correction, scratch.counts, scratch.pair, scratch.pair_weight, scratch.lists, scratch.token, scratch.weight, scratch.at],
                              [logits.stride(0), column, r.experts, r.top, r.groups, r.keep, int(r.softmax), int(r.normalized)], [r.scale, r.den_eps])
        self.n_up, self.n_down = up.n // r.experts, down.n // r.experts
        self.out = scratch.out

    @property
    def outputs(self) -> tuple:
        """Expert rows and where a token finds its own, as :func:`side_by_side` takes them."""
        o, r = self.out, self.spec.router
        return (o.data_ptr(), o.stride(0), int(o.dtype == torch.float32), self.s.at.data_ptr(), r.top, self.s.counts.data_ptr(), r.experts)

    def few(self, T: int) -> bool:
        """Whether the experts' weights are streamed for a few rows each, rather than multiplied in tiles behind a copy of the rows.
        On their own the tiles win from eight tokens on (unless the experts are so small that the copy's launch counts), but their
        CTAs take the SMs whole, and a decode step of that size does better with the mixer's kernels beside them."""
        r = self.spec.router
        chosen = min(r.experts, T * r.top) * (self.up.nbytes + self.down.nbytes) // r.experts
        return T * r.top <= self.s.pairs // 2 and (T <= 16 or (T <= FEW_ROWS and chosen < 48 << 20))

    def launches(self, T: int) -> int:
        return 2 + (1 if T <= lib().bonsai_lay_route_small(self.spec.router.top) and (self.s.exact or self.few(T)) else 2)

    def __call__(self, h: torch.Tensor, T: int, scratch: GemmScratch) -> None:
        l, s, st, r = lib(), self.s, K.stream(), self.spec.router
        pairs, hid = T * r.top, s.hidden[self.spec.ff]
        tile = not s.exact and not self.few(T)
        xs, chunks = (s.sorted, round_up(s.width, 8) // 8) if tile else (None, 0)
        K.check(l.bonsai_lay_route(*self.call.args, T, h.data_ptr(), h.stride(0), chunks, K.ptr(xs), 0 if xs is None else xs.stride(0), st), "route")
        lists, token, weight = s.lists.data_ptr(), s.token.data_ptr(), s.weight.data_ptr()
        up, down, g = self.up, self.down, self.glu
        if s.exact:
            self.out = s.out
            K.check(l.bonsai_lay_experts_f32(up.data.data_ptr(), r.experts, self.n_up, up.k, up.kp, h.data_ptr(), h.stride(0), lists, token, weight, pairs, T,
                                             hid.data_ptr(), hid.stride(0), 1, *g.args, st), "experts_f32")
            K.check(l.bonsai_lay_experts_f32(down.data.data_ptr(), r.experts, self.n_down, down.k, down.kp, hid.data_ptr(), hid.stride(0), lists, None, None,
                                             pairs, T, s.out.data_ptr(), s.out.stride(0), 0, *_NO_GLU.args, st), "experts_f32")
        elif not tile:
            self.out = s.out32
            slots, per = min(r.experts, pairs), min(T, 2 * pairs // r.experts + 8)
            K.check(l.bonsai_lay_experts_few(up.data.data_ptr(), r.experts, self.n_up, up.kp, h.data_ptr(), h.stride(0), lists, token, weight, pairs, slots, per,
                                             hid.data_ptr(), hid.stride(0), 1, *g.args, st), "experts_few")
            K.check(l.bonsai_lay_experts_few(down.data.data_ptr(), r.experts, self.n_down, down.kp, hid.data_ptr(), hid.stride(0), lists, None, None, pairs,
                                             slots, per, s.out32.data_ptr(), s.out32.stride(0), 0, *_NO_GLU.args, st), "experts_few")
        else:
            self.out = s.out
            wide = int(pairs > 96 * r.experts)
            K.check(l.bonsai_grouped_gemm_bf16(up.data.data_ptr(), r.experts, self.n_up, up.kp, xs.data_ptr(), xs.stride(0), pairs, lists, weight, hid.data_ptr(),
                                               hid.stride(0), 4, *g.args, wide, scratch.status.data_ptr(), scratch.sms, st), "grouped_gemm")
            K.check(l.bonsai_grouped_gemm_bf16(down.data.data_ptr(), r.experts, self.n_down, down.kp, hid.data_ptr(), hid.stride(0), pairs, lists, None,
                                               s.out.data_ptr(), s.out.stride(0), 6, *_NO_GLU.args, wide, scratch.status.data_ptr(), scratch.sms, st),
                    "grouped_gemm")


def sample(logits: torch.Tensor, *a, **kw) -> torch.Tensor:
    return K.sample(logits, *a, library=lib(), **kw)
