"""Front-ends of the hybrid decoder's kernels (``csrc/kernels/hybrid_rows.cu``, ``linear_scan.cu``, ``lightning_prefill.cu``,
``latent_*.cu``, ``gqa_attn.cu``, ``rglru.cu``, ``gemm_batched.cu``, ``gemm_f32.cu``).

GEMM operands are bf16, or fp32 in the 32-bit mode; the residual stream, norms, gates and states are fp32 in both.  A
projection's output reaches its consumer as bf16, as fp32, or as the fp32 workspace of a split-K GEMM that the consumer
leaves zero: ``Out`` carries the tensor together with that kind.
"""
from __future__ import annotations

import ctypes
import math
from dataclasses import dataclass

import torch

from . import _lib

vp, ci, cl, cf = ctypes.c_void_p, ctypes.c_int, ctypes.c_long, ctypes.c_float
SCAN_HGRN2, SCAN_WKV, SCAN_FIXED = 0, 1, 2
GATE_SILU, GATE_SIGMOID = 0, 1
ACTS = {"silu": 0, "relu": 1, "relu2": 2}       # relu2: the square of relu
KIND_BF16, KIND_F32, KIND_TAKE = 0, 1, 2
_sigs = {
    "artb_residual_step": [ci, vp, vp, ci, cl, vp, ci, ci, vp, vp, ci, vp, cf, vp, vp, vp, ci, ci, vp, vp, cl, vp, ci, ci, vp, vp, vp, cl, ci, vp, vp,
                           vp, ci, ci, ci, ci, cf, vp, vp, ci, ci, vp, vp, ci, ci, ci, vp],
    "artb_norm_shift_mix": [ci, vp, ci, vp, vp, ci, vp, cl, ci, vp, cl, vp, vp, vp, vp, ci, ci, ci, cf, vp, vp],
    "artb_poly_norm": [ci, vp, ci, ci, vp, vp, ci, ci, ci, ci, cf, vp],
    "artb_split_tanh": [ci, vp, ci, ci, vp, ci, ci, ci, ci, vp],
    "artb_gated_act": [ci, vp, ci, ci, vp, ci, ci, ci, ci, vp],
    "artb_plain_act": [ci, vp, ci, ci, vp, ci, ci, ci, ci, vp],
    "artb_head_norm": [ci, vp, ci, vp, ci, vp, ci, ci, ci, vp, ci, ci, ci, ci, ci, cf, vp],
    "artb_gather_norm": [ci, vp, ci, vp, ci, vp, vp, ci, ci, ci, cf, cl, vp, vp],
    "artb_linear_scan": [ci, vp, ci, vp, ci, vp, ci, ci, vp, ci, ci, vp, vp, vp, cl, ci, cl, vp, vp, vp, ci, ci, ci, ci, vp, ci, ci, vp, vp],
    "artb_linear_decode": [ci, ci, vp, ci, vp, ci, vp, ci, ci, vp, ci, ci, vp, vp, vp, cl, ci, cl, vp, vp, vp, ci, ci, ci, ci, vp, ci,
                           vp, ci, ci, vp, ci, ci, cf, vp, vp],
    "artb_lightning_prefill": [vp, vp, vp, ci, vp, vp, cl, ci, cl, vp, vp, vp, ci, ci, ci, ci, vp, ci, ci, vp, vp],
    "artb_latent_finish": [ci, vp, ci, ci, vp, vp, cf, ci, vp, vp, vp, ci, cl, ci, vp, vp, ci, vp, ci, ci, ci, ci, ci, ci, ci, ci, ci, cf, vp,
                           vp],
    "artb_latent_attend": [ci, vp, vp, ci, vp, ci, vp, ci, ci, cl, vp, vp, vp, ci, cf, vp, vp, ci, ci, ci, ci, vp, vp],
    "artb_latent_decode": [vp, vp, ci, vp, ci, vp, ci, ci, cl, vp, vp, vp, ci, cf, vp, vp, vp, ci, ci, ci, ci, ci, vp, vp],
    "artb_latent_gather": [vp, ci, vp, ci, ci, cl, vp, vp, vp, vp, ci, vp, ci, vp, vp],
    "artb_latent_prefill_tc": [vp, ci, ci, vp, ci, vp, ci, ci, vp, ci, ci, vp, vp, ci, vp, vp, vp, vp, ci, ci, cf, cf, cf, vp, ci, vp, ci, vp, ci, vp, ci, ci,
                               vp, ci, ci, ci, ci, ci, ci, ci, ci, vp, vp],
    "artb_latent_prefill": [vp, ci, vp, ci, vp, ci, ci, vp, vp, ci, vp, vp, vp, vp, ci, ci, cf, cf, cf, vp, ci, vp, ci, vp, ci, vp, ci, ci, vp, ci,
                            ci, ci, ci, ci, ci, ci, ci, vp],
    "artb_gqa_finish": [ci, vp, ci, ci, vp, vp, vp, ci, cl, vp, ci, ci, ci, ci, ci, ci, ci, ci, vp, vp],
    "artb_gqa_finish_norm": [ci, vp, ci, ci, vp, vp, vp, ci, cl, vp, ci, ci, ci, ci, ci, ci, ci, ci, vp, vp, ci, vp, cf, vp, cf, ci, ci, vp, vp, vp, ci, ci, vp,
                             vp],
    "artb_gqa_gather": [vp, ci, vp, ci, ci, cl, vp, vp, vp, vp, ci, ci, vp, vp, ci, ci, vp, vp],
    "artb_gqa_decode": [vp, ci, vp, ci, vp, ci, ci, cl, vp, vp, vp, ci, ci, cf, cf, cf, vp, ci, ci, vp, ci, vp, ci, ci, vp, ci, ci, vp, ci, ci, ci, ci, ci, ci, ci, vp, vp],
    "artb_gqa_attend": [ci, vp, ci, vp, ci, vp, ci, ci, cl, vp, vp, vp, ci, ci, cf, cf, cf, vp, ci, ci, vp, ci, vp, ci, ci, vp, ci, ci, ci, ci, ci, ci, ci, ci, vp, vp],
    "artb_short_conv": [ci, vp, ci, ci, vp, vp, vp, ci, vp, cl, vp, vp, vp, vp, ci, ci, vp, ci, ci, ci, ci, ci, ci, vp, vp],
    "artb_rglru": [ci, ci, vp, ci, ci, vp, ci, vp, vp, vp, vp, ci, ci, vp, vp, cl, vp, vp, vp, ci, vp, ci, cf, ci, ci, ci, ci, vp, vp],
    "artb_gemm_batched_bf16_tn": [vp, ci, ci, vp, ci, vp, ci, cl, ci, ci, ci, ci, ci, vp, vp],
    "artb_gemm_f32_tn": [vp, ci, cl, vp, ci, cl, vp, ci, cl, ci, ci, ci, ci, vp],
}
_bound: dict[str, object] = {}


def _f(name: str):
    fn = _bound.get(name)
    if fn is None:
        fn = getattr(_lib.kernels(), name)
        fn.argtypes, fn.restype = _sigs[name], ci
        _bound[name] = fn
    return fn


def pad(n: int, m: int = 8) -> int:
    return (n + m - 1) // m * m


@dataclass
class Out:
    """A projection's output as its consumer finds it: ``t`` [M, N] with unit inner stride and its kind."""
    t: torch.Tensor
    kind: int

    def col(self, c: int) -> "Out":
        return Out(self.t[:, c:], self.kind)


def as_out(t: torch.Tensor) -> Out:
    return Out(t, KIND_BF16 if t.dtype == torch.bfloat16 else KIND_F32)


def _is32(t: torch.Tensor) -> int:
    return 1 if t.dtype == torch.float32 else 0


def _st(t: torch.Tensor):
    return _lib.ptr(_lib.status_word(t.device))


@dataclass
class Sublayer:
    """What a sublayer hands to the residual stream: ``y`` (may be missing) times ``gate`` [M], ``bias`` [dp] and the rows of a
    token's experts, ``rows`` [cap, dp] weighted by ``weight`` [M, k] at the places ``pos`` [M, k]; a place of -1 is the token's
    row of ``identity``.  The sum is multiplied by the sigmoid of ``col_gate`` + ``col_bias`` [dp]."""
    y: Out | None = None
    bias: torch.Tensor | None = None
    rows: torch.Tensor | None = None
    pos: torch.Tensor | None = None
    weight: torch.Tensor | None = None
    gate: torch.Tensor | None = None
    identity: Out | None = None
    col_gate: Out | None = None
    col_bias: torch.Tensor | None = None


@dataclass
class Streams:
    """A boundary between hyper-connected sublayers: ``coef`` fp32 [(n_in + 2) * n_out] holds mix [n_in][n_out] (from, to), what each
    copy gets of the sublayer's result, and what the next sublayer takes of each copy.  ``n_in`` = 0: the embedding, all copies
    being equal to it."""
    n_in: int
    n_out: int
    coef: torch.Tensor


def residual_step(x_out: torch.Tensor, w_post: torch.Tensor | None, d: int, eps: float, *, y: Out | None = None, x_in=None,
                  mult: float = 1.0, tokens=None, table=None, sub: Sublayer | None = None, freq=None, pos=None, hist=None,
                  hist_n: int = 0, avg=None, w_next=None, h=None, streams: Streams | None = None) -> None:
    """One sublayer boundary of the fp32 residual stream ``[M, dp]``; ``y`` (or ``sub``) is the sublayer's output, or
    ``tokens`` / ``table`` the embedding, to which ``freq`` (fp64 ``[dp / 2]``) and ``pos`` add a sinusoidal position vector.
    ``w_post``: norm weight of the output; None: it is taken as it is, times ``mult``.  ``hist`` fp32 ``[layers + 1, M, dp]``: the result is stored at ``hist_n`` and, with ``avg``,
    replaced by the weighted average of entries ``0 .. hist_n``.  ``w_next`` / ``h``: the next sublayer's input norm; without
    ``w_next``, ``h`` is the stream itself in the operand dtype.  ``streams``: ``x_in`` and ``x_out`` hold several copies of the
    stream side by side, which the step mixes; ``h`` then comes from their weighted sum."""
    M, dp = x_out.shape
    if streams is not None:
        dp //= streams.n_out
        if streams.coef.numel() != (streams.n_in + 2) * streams.n_out or (x_in is not None and x_in.shape[1] != streams.n_in * dp):
            raise ValueError("streams: the tensors do not hold as many copies as the boundary has")
    cg = sub.col_gate if sub is not None else None
    s = sub if sub is not None else Sublayer(y)
    y, ex = s.y, s.rows
    idn = s.identity
    op = next((t for t in (table, h, ex) if t is not None), None)      # any tensor of the operand dtype
    f32 = _is32(op) if op is not None else 0
    if freq is not None and freq.dtype != torch.float64:
        raise ValueError("position frequencies are fp64")
    _lib.check_rc(_f("artb_residual_step")(
        f32, _lib.ptr(tokens), _lib.ptr(table), table.stride(0) if table is not None else 0, table.shape[0] if table is not None else 0,
        _lib.ptr(y.t if y is not None else None), y.t.stride(0) if y is not None else 0, y.kind if y is not None else 0,
        _lib.ptr(x_in), _lib.ptr(x_out), x_out.stride(0), _lib.ptr(w_post), mult, _lib.ptr(s.gate), _lib.ptr(s.bias), _lib.ptr(ex),
        ex.stride(0) if ex is not None else 0, s.pos.shape[1] if ex is not None else 0, _lib.ptr(s.pos), _lib.ptr(s.weight),
        ex.shape[0] if ex is not None else 0, _lib.ptr(idn.t if idn is not None else None), idn.t.stride(0) if idn is not None else 0,
        idn.kind if idn is not None else 0, _lib.ptr(freq), _lib.ptr(pos), _lib.ptr(hist),
        hist.stride(0) if hist is not None else 0, hist_n, _lib.ptr(avg), _lib.ptr(w_next), _lib.ptr(h),
        h.stride(0) if h is not None else 0, M, d, dp, eps, _st(x_out), _lib.ptr(cg.t if cg is not None else None), cg.t.stride(0) if cg is not None else 0,
        cg.kind if cg is not None else 0, _lib.ptr(s.col_bias), _lib.ptr(streams.coef if streams else None), streams.n_in if streams else 0,
        streams.n_out if streams else 0, x_in.stride(0) if streams and x_in is not None else 0, _lib.stream_ptr()), "residual_step")


def norm_shift_mix(x, w, mu, out, state, row_seq, cu_q, ctx, state_slot, d: int, eps: float) -> None:
    """``out[s, m] = h + (h' - h) mu[s]`` with ``h`` the normed row and ``h'`` that of the token before it; ``out`` is
    ``[n_mix, pitch, dp]``, ``state`` fp32 ``[slots, dp]``."""
    M, dp = x.shape
    _lib.check_rc(_f("artb_norm_shift_mix")(
        _is32(out), _lib.ptr(x), x.stride(0), _lib.ptr(w), _lib.ptr(mu), mu.shape[0], _lib.ptr(out), out.stride(0), out.stride(1),
        _lib.ptr(state), state.shape[0], _lib.ptr(row_seq), _lib.ptr(cu_q), _lib.ptr(ctx), _lib.ptr(state_slot), M, d, dp, eps,
        _st(x), _lib.stream_ptr()), "norm_shift_mix")


def poly_norm(z: Out, act, out, n: int, eps: float) -> torch.Tensor:
    _lib.check_rc(_f("artb_poly_norm")(_is32(out), _lib.ptr(z.t), z.t.stride(0), z.kind, _lib.ptr(act), _lib.ptr(out), out.stride(0),
                                       out.shape[0], n, out.shape[1], eps, _lib.stream_ptr()), "poly_norm")
    return out


def split_tanh(z: Out, r: int, rp: int, out) -> torch.Tensor:
    """bf16 ``[M, 2 rp]``: tanh of the first ``r`` columns as a pair of bf16 values; fp32 ``[M, rp]``: tanh."""
    _lib.check_rc(_f("artb_split_tanh")(_is32(out), _lib.ptr(z.t), z.t.stride(0), z.kind, _lib.ptr(out), out.stride(0), out.shape[0],
                                        r, rp, _lib.stream_ptr()), "split_tanh")
    return out


def gated_act(z: Out, out, act: str) -> torch.Tensor:
    """``act(gate) * up`` of a gate|up projection whose columns are interleaved in blocks of 16."""
    _lib.check_rc(_f("artb_gated_act")(_is32(out), _lib.ptr(z.t), z.t.stride(0), z.kind, _lib.ptr(out), out.stride(0), out.shape[0],
                                       out.shape[1], ACTS[act], _lib.stream_ptr()), "gated_act")
    return out


def plain_act(z: Out, out, act: str) -> torch.Tensor:
    """``act(z)``, for a consumer behind a split product."""
    _lib.check_rc(_f("artb_plain_act")(_is32(out), _lib.ptr(z.t), z.t.stride(0), z.kind, _lib.ptr(out), out.stride(0), out.shape[0],
                                       out.shape[1], ACTS[act], _lib.stream_ptr()), "plain_act")
    return out


def head_norm(o, w, w_per_head: bool, H: int, vdim: int, vpad: int, out, eps: float, gate: Out | None = None,
              gate_act: int = GATE_SILU) -> torch.Tensor:
    """Per-head RMSNorm of ``o`` fp32 [M, H * vdim]; ``w`` [vdim], or [H * vdim] with ``w_per_head``; silu or sigmoid ``gate``.
    H = 1: one norm over the whole row."""
    _lib.check_rc(_f("artb_head_norm")(
        _is32(out), _lib.ptr(o), o.stride(0), _lib.ptr(w), 1 if w_per_head else 0,
        _lib.ptr(gate.t if gate else None), gate.t.stride(0) if gate else 0, gate.kind if gate else 0, gate_act, _lib.ptr(out),
        out.stride(0), out.shape[0], H, vdim, vpad, eps, _lib.stream_ptr()), "head_norm")
    return out


def gather_norm(x, rows, w, h, d: int, eps: float) -> torch.Tensor:
    _lib.check_rc(_f("artb_gather_norm")(_is32(h), _lib.ptr(x), x.stride(0), _lib.ptr(rows), rows.numel(), _lib.ptr(w), _lib.ptr(h),
                                         h.stride(0), d, x.shape[1], eps, x.shape[0], _st(x), _lib.stream_ptr()), "gather_norm")
    return h


def _scan_in(mode, q: Out, k: Out | None, v: Out, g: Out | None):
    if q.kind != v.kind or (k is not None and k.kind != q.kind):
        raise ValueError("q, k and v come from one projection and share their kind")
    return (_lib.ptr(q.t), q.t.stride(0), _lib.ptr(k.t if k else None), k.t.stride(0) if k else 0, _lib.ptr(v.t), v.t.stride(0), q.kind,
            _lib.ptr(g.t if g else None), g.t.stride(0) if g else 0, g.kind if g else KIND_F32)


def linear_scan(mode: int, q: Out, k: Out | None, v: Out, g: Out | None, bias, aux, state, cu_q, ctx, state_slot, n_seqs: int, H: int,
                dim: int, vdim: int, o) -> torch.Tensor:
    """Portions of ``n_seqs`` sequences through the recurrence; ``state`` fp32 ``[slots, H, vdim, ld]``; ``o`` fp32."""
    _lib.check_rc(_f("artb_linear_scan")(
        mode, *_scan_in(mode, q, k, v, g), _lib.ptr(bias), _lib.ptr(aux), _lib.ptr(state), state.stride(0), state.shape[3],
        state.shape[0], _lib.ptr(cu_q), _lib.ptr(ctx), _lib.ptr(state_slot), n_seqs, H, dim, vdim, _lib.ptr(o), o.stride(0),
        o.shape[0], _st(o),
        _lib.stream_ptr()), "linear_scan")
    return o


def linear_decode(mode: int, q: Out, k: Out | None, v: Out, g: Out | None, bias, aux, state, cu_q, ctx, state_slot, H: int, dim: int,
                  vdim: int, w, w_per_head: bool, gate: Out | None, out, vpad: int, eps: float) -> torch.Tensor:
    """One token of each sequence (row m = sequence m): recurrence, per-head norm, optional gate.  ``w`` None: the fp32 outputs
    of the recurrence."""
    M = out.shape[0]
    _lib.check_rc(_f("artb_linear_decode")(
        _is32(out) if w is not None else 0, mode, *_scan_in(mode, q, k, v, g), _lib.ptr(bias), _lib.ptr(aux), _lib.ptr(state), state.stride(0),
        state.shape[3], state.shape[0], _lib.ptr(cu_q), _lib.ptr(ctx), _lib.ptr(state_slot), M, H, dim, vdim, _lib.ptr(w),
        1 if w_per_head else 0, _lib.ptr(gate.t if gate else None), gate.t.stride(0) if gate else 0, gate.kind if gate else 0,
        _lib.ptr(out), out.stride(0), vpad, eps, _st(out), _lib.stream_ptr()), "linear_decode")
    return out


def lightning_tc(dim: int, vdim: int) -> bool:
    """Whether the tensor-core form of lightning attention takes these head sizes."""
    return dim <= 128 and dim % 8 == 0 and vdim % 8 == 0


def lightning_prefill(q, k, v, decay, state, cu_q, ctx, state_slot, n_seqs: int, H: int, dim: int, vdim: int, o) -> torch.Tensor:
    """``linear_scan(SCAN_FIXED, ...)`` in chunks on tensor cores; ``q``, ``k``, ``v`` bf16 columns of one projection that have
    been through the silu already."""
    if not q.stride(0) == k.stride(0) == v.stride(0):
        raise ValueError("q, k and v come from one projection")
    _lib.check_rc(_f("artb_lightning_prefill")(
        _lib.ptr(q), _lib.ptr(k), _lib.ptr(v), q.stride(0), _lib.ptr(decay), _lib.ptr(state), state.stride(0), state.shape[3], state.shape[0],
        _lib.ptr(cu_q), _lib.ptr(ctx), _lib.ptr(state_slot), n_seqs, H, dim, vdim, _lib.ptr(o), o.stride(0), o.shape[0], _st(o),
        _lib.stream_ptr()), "lightning_prefill")
    return o


@dataclass
class Rotation:
    """The rotation of the first ``dims`` columns of a head (or of its rotated part): ``freq`` fp64 [dims / 2] per pair (on the device),
    ``scale`` the factor of sine and cosine; a column's partner is its neighbour (``next``) or ``dims / 2`` columns further."""
    dims: int
    freq: torch.Tensor
    scale: float = 1.0
    next: bool = False


def _rotation(rot: Rotation | None) -> None:
    if rot is not None and (rot.freq.dtype != torch.float64 or rot.freq.numel() != rot.dims // 2):
        raise ValueError("rotation frequencies are fp64, one per pair")


def latent_finish(p: Out, w, rotation: Rotation, pos, slot, cache, n_abs: int, qn, qr, qe, H: int, dim: int, rank: int, eps: float) -> None:
    """Norm, rotation and cache write behind the q | latent projection.  Rows below ``n_abs`` leave their queries in
    ``qn`` [H, pitch, dim_p] / ``qr`` [H, pitch, rot_p], the others in ``qe`` [M - n_abs, H * (dim_p + rot_p)]."""
    M, rot = pos.numel(), rotation.dims
    _rotation(rotation)
    _lib.check_rc(_f("artb_latent_finish")(
        _is32(cache), _lib.ptr(p.t), p.t.stride(0), p.kind, _lib.ptr(w), _lib.ptr(rotation.freq), rotation.scale, int(rotation.next), _lib.ptr(pos), _lib.ptr(slot),
        _lib.ptr(cache), cache.shape[-1], cache.shape[0] * cache.shape[1], n_abs, _lib.ptr(qn), _lib.ptr(qr),
        qn.shape[1] if qn is not None else 0, _lib.ptr(qe), qe.stride(0) if qe is not None else 0, M, H, dim, pad(dim, 16), rot,
        pad(rot, 16), rank, pad(rank, 16), eps, _st(cache), _lib.stream_ptr()), "latent_finish")


def latent_attend(ql, qr, cache, block_table, row_seq, pos, ctx, window: int, scale: float, o, M: int, sink=None) -> torch.Tensor:
    """Windowed attention in latent space over the paged cache, scalar fp32 form; everything head-major [H, pitch, .].  ``sink`` fp32
    [H]: one more term of the softmax's denominator."""
    H, pitch, rank_p = ql.shape
    _lib.check_rc(_f("artb_latent_attend")(
        _is32(cache), _lib.ptr(ql), _lib.ptr(qr), pitch, _lib.ptr(cache), cache.shape[-1], _lib.ptr(block_table),
        block_table.stride(0), cache.shape[1], cache.shape[0], _lib.ptr(row_seq), _lib.ptr(pos), _lib.ptr(ctx), window, scale,
        _lib.ptr(sink), _lib.ptr(o), M, H, rank_p, qr.shape[2], _st(cache), _lib.stream_ptr()), "latent_attend")
    return o


LATENT_TILE = 64        # keys per tile of the decode kernel: the unit its splits are made of
PREFILL_ROWS = 128      # query rows per CTA of the prefill kernel


def latent_decode_splits(M: int, H: int, keys: int, sms: int = 148) -> int:
    """How many CTAs share a token's window: enough to cover the machine, two tiles each at least."""
    ctas = M * ((H + 31) // 32 if H > 16 else 1)
    return max(1, min(sms // max(1, ctas), (keys + LATENT_TILE - 1) // LATENT_TILE // 2, 32))


def latent_decode(ql, qr, cache, block_table, row_seq, pos, ctx, window: int, scale: float, o, M: int, splits: int = 1,
                  ws=None, sink=None) -> torch.Tensor:
    """Tensor-core form of :func:`latent_attend` for rows ``0 .. M - 1`` (bf16)."""
    H, pitch, rank_p = ql.shape
    if splits > 1 and ws is None:
        ws = torch.empty(M * H * splits * (rank_p + 2), dtype=torch.float32, device=o.device)
    _lib.check_rc(_f("artb_latent_decode")(
        _lib.ptr(ql), _lib.ptr(qr), pitch, _lib.ptr(cache), cache.shape[-1], _lib.ptr(block_table), block_table.stride(0),
        cache.shape[1], cache.shape[0], _lib.ptr(row_seq), _lib.ptr(pos), _lib.ptr(ctx), window, scale, _lib.ptr(sink), _lib.ptr(o), _lib.ptr(ws), splits,
        M, H, rank_p, qr.shape[2], _st(cache), _lib.stream_ptr()), "latent_decode")
    return o


@dataclass
class PrefillPlan:
    """Query tiles and gathered key ranges of the portions of one batch under one window (int32, on the device).  Row
    numbers count from the first portion row of the batch."""
    n_keys: int
    n_tiles: int
    n_seqs: int
    seq_of: torch.Tensor
    key_off: torch.Tensor
    key_pos0: torch.Tensor
    key_cnt: torch.Tensor
    row_end: torch.Tensor
    row_pos0: torch.Tensor
    tile_seq: torch.Tensor
    tile_row: torch.Tensor


def first_key(p: int, window: int, chunk: int = 0) -> int:
    """First key position ``p`` sees: of the last ``window`` ones and of its own ``chunk`` (0: no limit)."""
    lo = max(0, p - window + 1) if window > 0 else 0
    return max(lo, p - p % chunk) if chunk > 0 else lo


def plan_prefill(portions: list[tuple[int, int, int]], window: int, device, chunk: int = 0) -> PrefillPlan:
    """``portions``: ``(sequence, tokens before the portion, tokens of the portion)`` in row order.  Every sequence's
    gathered keys start at a multiple of 8 rows."""
    seq_of, key_off, key_pos0, key_cnt, row_end, row_pos0, tile_seq, tile_row = [], [], [], [], [], [], [], []
    row = keys = 0
    for i, (seq, n0, n) in enumerate(portions):
        first = first_key(n0, window, chunk)
        seq_of.append(seq)
        key_off.append(keys)
        key_pos0.append(first)
        key_cnt.append(n0 + n - first)
        keys += pad(n0 + n - first)
        row_pos0.append(n0 - row)
        for r in range(row, row + n, PREFILL_ROWS):
            tile_seq.append(i)
            tile_row.append(r)
        row += n
        row_end.append(row)
    t = lambda v: torch.tensor(v, dtype=torch.int32, device=device)      # noqa: E731
    return PrefillPlan(keys, len(tile_seq), len(portions), t(seq_of), t(key_off), t(key_pos0), t(key_cnt), t(row_end), t(row_pos0), t(tile_seq), t(tile_row))


def latent_gather(cache, block_table, plan: PrefillPlan) -> torch.Tensor:
    """The cache rows the portions' windows reach, contiguous: ``[n_keys, rank_p + rot_p]``."""
    out = torch.empty((plan.n_keys, cache.shape[-1]), dtype=cache.dtype, device=cache.device)
    _lib.check_rc(_f("artb_latent_gather")(
        _lib.ptr(cache), cache.shape[-1], _lib.ptr(block_table), block_table.stride(0), cache.shape[1], cache.shape[0],
        _lib.ptr(plan.seq_of), _lib.ptr(plan.key_off), _lib.ptr(plan.key_pos0), _lib.ptr(plan.key_cnt), plan.n_seqs, _lib.ptr(out), plan.n_keys, _st(cache),
        _lib.stream_ptr()), "latent_gather")
    return out


def _gate(gate):
    return _lib.ptr(gate), gate.stride(0) if gate is not None else 0


BIAS_PAD = 256          # entries in front of and behind a distance table (key_weights.cuh)


@dataclass
class KeyWeights:
    """What an attention kernel makes of scores besides a softmax, and of its result.  ``bias`` fp32 [H, n + 2 BIAS_PAD] (see
    :func:`distance_table`): a key weighs sigmoid(score + bias of its distance), without normalisation.  ``sink`` fp32 [H]: one
    more term of the softmax's denominator.  ``cols`` [rows, .], operand dtype: logits of a gate of the result's columns, a head's
    ``pitch`` columns after the one before it."""
    bias: torch.Tensor | None = None
    sink: torch.Tensor | None = None
    cols: torch.Tensor | None = None
    pitch: int = 0

    def rows_from(self, n: int) -> "KeyWeights":
        """The same for the rows from ``n`` on."""
        return KeyWeights(self.bias, self.sink, self.cols[n:] if self.cols is not None else None, self.pitch)


def distance_table(rel: torch.Tensor, buckets: list[int], head_bias: torch.Tensor) -> torch.Tensor:
    """The kernels' table of ``rel`` fp32 [rows, H] by distance plus ``head_bias`` [H], in base-2 units; ``buckets[t]`` is the row of
    distance t, the last one that of all farther ones."""
    idx = torch.tensor([buckets[0]] * BIAS_PAD + list(buckets) + [buckets[-1]] * BIAS_PAD, device=rel.device)
    return ((rel.double()[idx] + head_bias.double()) * math.log2(math.e)).t().float().contiguous()


def _bias(kw: "KeyWeights | None", H: int):
    b = kw.bias if kw is not None else None
    if b is not None and (b.dtype != torch.float32 or b.shape[0] != H or not b.is_contiguous() or b.shape[1] <= 2 * BIAS_PAD):
        raise ValueError("a distance table is fp32 [heads, distances + padding]")
    return (1, _lib.ptr(b), b.shape[1] - 2 * BIAS_PAD) if b is not None else (0, _lib.ptr(None), 0)


def _cols(kw: "KeyWeights | None", like: torch.Tensor):
    c = kw.cols if kw is not None else None
    if c is not None and (c.dtype != like.dtype or c.stride(1) != 1):
        raise ValueError("a column gate has the operand dtype and unit inner stride")
    return _lib.ptr(c), c.stride(0) if c is not None else 0, kw.pitch if kw is not None else 0


def latent_prefill(q, kv, c, plan: PrefillPlan, window: int, scale: float, o, H: int, dk: int, dv: int, rank_p: int, rot_p: int,
                   vdim: int, chunk: int = 0, G: int = 1, out_scale: float = 1.0, softcap: float = 0.0, gate=None,
                   weights: KeyWeights | None = None) -> torch.Tensor:
    """Masked attention of the portions: ``q`` [rows, H * (dk + rot_p)], ``kv`` [n_keys, H / G * (dk + dv)] the expanded
    keys and values (``G`` heads share them), ``c`` the gathered cache rows; ``o`` [rows, H * pad(vdim)].  ``softcap`` > 0 squashes
    the scores; ``gate`` fp32 [rows, H] multiplies the heads."""
    _lib.check_rc(_f("artb_latent_prefill")(
        _lib.ptr(q), q.stride(0), _lib.ptr(kv), kv.stride(0), _lib.ptr(c), c.stride(0), rank_p, _lib.ptr(plan.tile_seq),
        _lib.ptr(plan.tile_row), plan.n_tiles, _lib.ptr(plan.row_end), _lib.ptr(plan.row_pos0), _lib.ptr(plan.key_off),
        _lib.ptr(plan.key_pos0), window, chunk, scale, softcap, out_scale, *_gate(gate), _lib.ptr(weights.sink if weights else None), *_bias(weights, H),
        *_cols(weights, o), _lib.ptr(o), o.stride(0), pad(vdim), vdim, H, G, dk, dv, rot_p,
        _lib.stream_ptr()), "latent_prefill")
    return o


def prefill_tc_values(dim: int, rot: int, vdim: int, scale: float) -> int:
    """Value columns per head the tcgen05 prefill kernel would use (0: the sizes do not suit it)."""
    if dim % 64 or rot % 64 or dim + rot > 192 or vdim > 128 or scale <= 0:
        return 0
    return 64 if vdim <= 64 else 128


def gqa_value_columns(dim: int, vdim: int, scale: float) -> int:
    """Columns of a value head in the cache of grouped-query attention: what the prefill kernel that suits the sizes reads."""
    return prefill_tc_values(dim, 0, vdim, scale) or pad(vdim, 16)


def latent_prefill_tc(q, k, vt, c, plan: PrefillPlan, window: int, scale: float, o, H: int, dk: int, dv: int, rank_p: int, rot_p: int,
                      vdim: int, chunk: int = 0, G: int = 1, out_scale: float = 1.0, softcap: float = 0.0, gate=None,
                      weights: KeyWeights | None = None) -> torch.Tensor:
    """:func:`latent_prefill` on tcgen05: ``k`` [n_keys, H / G * dk], values transposed ``vt`` [H / G * dv, n_keys]."""
    _lib.check_rc(_f("artb_latent_prefill_tc")(
        _lib.ptr(q), q.stride(0), q.shape[0], _lib.ptr(k), k.stride(0), _lib.ptr(c), c.stride(0), rank_p, _lib.ptr(vt), vt.stride(0),
        plan.n_keys, _lib.ptr(plan.tile_seq), _lib.ptr(plan.tile_row), plan.n_tiles, _lib.ptr(plan.row_end), _lib.ptr(plan.row_pos0),
        _lib.ptr(plan.key_off), _lib.ptr(plan.key_pos0), window, chunk, scale, softcap, out_scale, *_gate(gate), _lib.ptr(weights.sink if weights else None),
        *_bias(weights, H), *_cols(weights, o), _lib.ptr(o), o.stride(0), pad(vdim), vdim, H, G, dk, dv, rot_p, _st(o),
        _lib.stream_ptr()), "latent_prefill_tc")
    return o


def gqa_finish(p: Out, bias, slot, cache, q, H: int, Hkv: int, dim: int, vdim: int, dvp: int) -> None:
    """Biases, cache write and padded queries behind a q | k | v projection; cache rows hold ``Hkv`` keys of pad(dim, 16), then
    ``Hkv`` values of ``dvp`` columns."""
    M = slot.numel()
    _lib.check_rc(_f("artb_gqa_finish")(
        _is32(cache), _lib.ptr(p.t), p.t.stride(0), p.kind, _lib.ptr(bias), _lib.ptr(slot), _lib.ptr(cache), cache.shape[-1],
        cache.shape[0] * cache.shape[1], _lib.ptr(q), q.stride(0), M, H, Hkv, dim, pad(dim, 16), vdim, dvp, _st(cache), _lib.stream_ptr()),
        "gqa_finish")


def gqa_finish_norm(p: Out, bias, slot, cache, q, H: int, Hkv: int, dim: int, vdim: int, dvp: int, wq, wk, eps: float, rot: Rotation | None, pos,
                    gate=None, per_head: bool = False, q_scale=None, cols=None, pitch: int = 0) -> None:
    """:func:`gqa_finish` with norms over all heads of q (``wq``) and of k (``wk``), a rotation behind them, and ``gate`` fp32 [M, H]
    receiving the sigmoids of the columns behind v.  ``Hkv`` = 0: the projection has no k and v and the cache stays as it is.

    ``per_head``: a norm over each head with the weights of one; ``q_scale`` fp32 [H] then multiplies the query heads.  ``cols``
    [M, H * pitch], operand dtype: receives the ``H * vdim`` columns behind v."""
    M = slot.numel()
    _rotation(rot)
    if per_head and any(w is not None and w.numel() != dim for w in (wq, wk)):
        raise ValueError("per_head: norm weights of one head")
    if cols is not None and cols.dtype != q.dtype:
        raise ValueError("cols: a tensor of the operand dtype")
    if gate is not None and gate.stride(0) != H:
        raise ValueError("gate: a dense [M, H] tensor")
    _lib.check_rc(_f("artb_gqa_finish_norm")(
        _is32(cache), _lib.ptr(p.t), p.t.stride(0), p.kind, _lib.ptr(bias), _lib.ptr(slot), _lib.ptr(cache), cache.shape[-1],
        cache.shape[0] * cache.shape[1], _lib.ptr(q), q.stride(0), M, H, Hkv, dim, pad(dim, 16), vdim, dvp, _lib.ptr(wq), _lib.ptr(wk), int(per_head),
        _lib.ptr(q_scale), eps, _lib.ptr(rot.freq if rot else None), rot.scale if rot else 1.0, rot.dims if rot else 0, 1 if rot and rot.next else 0, _lib.ptr(pos),
        _lib.ptr(gate), _lib.ptr(cols), cols.stride(0) if cols is not None else 0, pitch, _st(cache), _lib.stream_ptr()), "gqa_finish_norm")


def gqa_gather(cache, block_table, plan: PrefillPlan, Hkv: int, dk: int, dv: int) -> tuple[torch.Tensor, torch.Tensor]:
    """Keys ``[n_keys, Hkv * dk]`` and transposed values ``[Hkv * dv, n_keys]`` of the cache rows the portions see."""
    k = torch.empty((plan.n_keys, Hkv * dk), dtype=cache.dtype, device=cache.device)
    vt = torch.empty((Hkv * dv, plan.n_keys), dtype=cache.dtype, device=cache.device)
    _lib.check_rc(_f("artb_gqa_gather")(
        _lib.ptr(cache), cache.shape[-1], _lib.ptr(block_table), block_table.stride(0), cache.shape[1], cache.shape[0],
        _lib.ptr(plan.seq_of), _lib.ptr(plan.key_off), _lib.ptr(plan.key_pos0), _lib.ptr(plan.key_cnt), plan.n_seqs, plan.n_keys, _lib.ptr(k),
        _lib.ptr(vt), Hkv * dk, Hkv * dv, _st(cache), _lib.stream_ptr()), "gqa_gather")
    return k, vt


GQA_TILE = 32           # keys per warp tile of the decode kernel, four warps a CTA
GQA_DECODE_MAX = 256    # head sizes its tiles hold; beyond them the scalar kernel serves


def gqa_decode_splits(M: int, ctas_per_row: int, keys: int, sms: int = 148) -> int:
    """How many CTAs share a row's keys: enough to cover the machine, one tile per warp each at least."""
    return max(1, min(2 * sms // max(1, M * ctas_per_row), (keys + 4 * GQA_TILE - 1) // (4 * GQA_TILE), 32))


def _gqa(q, cache, block_table, row_seq, pos, ctx, window, chunk, scale, out_scale, o, softcap, gate, weights, H):
    if weights is not None and weights.sink is not None:
        raise ValueError("sinks are not supported by this form of attention")
    return (_lib.ptr(q), q.stride(0), _lib.ptr(cache), cache.shape[-1], _lib.ptr(block_table), block_table.stride(0), cache.shape[1],
            cache.shape[0], _lib.ptr(row_seq), _lib.ptr(pos), _lib.ptr(ctx), window, chunk, scale, softcap, out_scale, *_gate(gate),
            *_bias(weights, H), *_cols(weights, o), _lib.ptr(o), o.stride(0))


def gqa_decode(q, cache, block_table, row_seq, pos, ctx, window: int, chunk: int, scale: float, out_scale: float, o, M: int, H: int,
               Hkv: int, dim: int, vdim: int, dvp: int, splits: int = 1, softcap: float = 0.0, gate=None,
               weights: KeyWeights | None = None) -> torch.Tensor:
    """Rows ``0 .. M - 1`` of ``q`` against their sequences' cached keys; ``o`` [., H * pad(vdim)] gets ``out_scale`` times the
    result, and times ``gate`` fp32 [M, H]; ``softcap`` > 0 squashes the scores."""
    vpad = pad(vdim)
    ws = torch.empty(M * H * splits * (vpad + 2), dtype=torch.float32, device=o.device) if splits > 1 else None
    _lib.check_rc(_f("artb_gqa_decode")(
        *_gqa(q, cache, block_table, row_seq, pos, ctx, window, chunk, scale, out_scale, o, softcap, gate, weights, H), vpad, _lib.ptr(ws), splits, M, H, Hkv,
        pad(dim, 16), vdim, dvp, _st(cache), _lib.stream_ptr()), "gqa_decode")
    return o


def gqa_attend(q, cache, block_table, row_seq, pos, ctx, window: int, chunk: int, scale: float, out_scale: float, o, M: int, H: int,
               Hkv: int, dim: int, vdim: int, dvp: int, softcap: float = 0.0, gate=None, weights: KeyWeights | None = None) -> torch.Tensor:
    """Scalar fp32 form of :func:`gqa_decode`, any head sizes."""
    _lib.check_rc(_f("artb_gqa_attend")(
        _is32(cache), *_gqa(q, cache, block_table, row_seq, pos, ctx, window, chunk, scale, out_scale, o, softcap, gate, weights, H), pad(vdim), M, H, Hkv,
        pad(dim, 16), vdim, dvp, _st(cache), _lib.stream_ptr()), "gqa_attend")
    return o


def short_conv(x: Out, x_bias, w, bias, state, row_seq, cu_q, ctx, state_slot, n_seqs: int, single: bool, u, bs: int, bp: int) -> None:
    """Causal convolution ``w`` [n, taps] of ``x + x_bias``; ``u`` [blocks, pitch, .] receives a bf16 pair (or fp32) per
    channel, ``state`` fp32 [slots, taps - 1, n] the last inputs."""
    n, taps = w.shape
    _lib.check_rc(_f("artb_short_conv")(
        _is32(u), _lib.ptr(x.t), x.t.stride(0), x.kind, _lib.ptr(x_bias), _lib.ptr(w), _lib.ptr(bias), taps, _lib.ptr(state),
        state.shape[0], _lib.ptr(row_seq), _lib.ptr(cu_q), _lib.ptr(ctx), _lib.ptr(state_slot), n_seqs, 1 if single else 0, _lib.ptr(u),
        u.shape[1], u.shape[2], n, bs, bp, x.t.shape[0], _st(u), _lib.stream_ptr()), "short_conv")


def rglru(u, z, r_bias, i_bias, decay, y: Out, y_bias, state, cu_q, ctx, state_slot, n_seqs: int, single: bool, o, out_scale: float,
          bs: int, bp: int) -> None:
    """Gated recurrence over ``u`` (see :func:`short_conv`) with gate products ``z`` fp32 [M, blocks * 2 bp]; ``o`` [M, n] gets
    ``out_scale * S * gelu(y + y_bias)``."""
    n = decay.numel()
    _lib.check_rc(_f("artb_rglru")(
        _is32(u), 1 if single else 0, _lib.ptr(u), u.shape[1], u.shape[2], _lib.ptr(z), z.stride(0), _lib.ptr(r_bias), _lib.ptr(i_bias),
        _lib.ptr(decay), _lib.ptr(y.t), y.t.stride(0), y.kind, _lib.ptr(y_bias), _lib.ptr(state), state.shape[0], _lib.ptr(cu_q),
        _lib.ptr(ctx), _lib.ptr(state_slot), n_seqs, _lib.ptr(o), o.stride(0), out_scale, n, bs, bp, z.shape[0], _st(u), _lib.stream_ptr()),
        "rglru")


def gemm_batched(a, b, out, M: int, *, c_batch: int) -> torch.Tensor:
    """``out_b[m, n] = a[b, m, :] . b[b, n, :]``; ``a`` [batch, pitch, K], ``b`` [batch, N, K]; ``out`` is a 2-D tensor whose
    storage receives member ``b`` from element ``b * c_batch`` on (leading dimension ``out.stride(0)``)."""
    batch, pitch, K = a.shape
    N = b.shape[1]
    if a.dtype == torch.float32:
        _lib.check_rc(_f("artb_gemm_f32_tn")(_lib.ptr(a), a.stride(1), a.stride(0), _lib.ptr(b), b.stride(1), b.stride(0), _lib.ptr(out),
                                             out.stride(0), c_batch, batch, M, N, K, _lib.stream_ptr()), "gemm_f32")
        return out
    if not (a.is_contiguous() and b.is_contiguous()):
        raise ValueError("batched operands must be contiguous")
    _lib.check_rc(_f("artb_gemm_batched_bf16_tn")(_lib.ptr(a), a.stride(1), pitch, _lib.ptr(b), b.stride(1), _lib.ptr(out), out.stride(0),
                                                  c_batch, _is32(out), batch, M, N, K, _st(a), _lib.stream_ptr()), "gemm_batched")
    return out


def gemm_f32(a, b, out=None) -> torch.Tensor:
    """``out[M, N] = a[M, K] @ b[N, K].T`` in fp32 multiply-adds (no reduced-precision mode)."""
    if a.dtype != torch.float32 or b.dtype != torch.float32 or a.stride(1) != 1 or b.stride(1) != 1:
        raise ValueError("gemm_f32: fp32 operands with unit inner stride")
    M, K = a.shape
    N = b.shape[0]
    if out is None:
        out = torch.empty((M, N), dtype=torch.float32, device=a.device)
    _lib.check_rc(_f("artb_gemm_f32_tn")(_lib.ptr(a), a.stride(0), 0, _lib.ptr(b), b.stride(0), 0, _lib.ptr(out), out.stride(0), 0, 1, M, N,
                                         K, _lib.stream_ptr()), "gemm_f32")
    return out
