"""Ops of the layered decoders (mixers, experts, 32-bit residual stream): CUDA tensors go to the sm_100a
kernels, CPU tensors to the PyTorch statements in ``mixer_torch``.  Activations are bf16 (serving) or fp32 (a model run
in 32-bit); the residual stream, scores, norms and recurrent states are fp32 either way.

Matrices whose rows are read by TMA have a row pitch that is a multiple of 8 elements (``rows_buffer``,
``padded_weight``), so no width has to be."""
from __future__ import annotations

import ctypes
from dataclasses import dataclass
from typing import NamedTuple

import torch

from . import mixer_torch, native
from .native import _check, _ptr, _req, _stream

TILE = 128                 # rows of an expert tile (csrc/mixer_elementwise.cu: PLAN_TILE)
_declared = False


def _lib():
    global _declared
    lib = native.load()
    if not _declared:
        P, I, L, F = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong, ctypes.c_float
        for name, args in {
            "b200_residual_norm": [P, P, I, F, P, P, P, P, F, P, L, F, P, P, I, I, L, I, I, I, I, P, P],
            "b200_moe_plan": [P, P, I, I, I, P, P, P, P, L, P, I, P, P],
            "b200_moe_plan_layers": [],
            "b200_add_normed": [P, P, I, P, P, L, P, P, L, F, I, I, I, P, P],
            "b200_glu_any": [P, P, L, I, L, L, I, I, P],
            "b200_gate_sigmoid": [P, P, L, I, I, L, L, I, P],
            "b200_gemm_f32": [P, P, P, I, I, I, L, L, L, I, P, I, I, I, I, P, P],
            "b200_gemm_bf16_grouped": [P, P, P, P, I, I, I, L, L, L, L, P, I, I, I, I, I, I, I, I, P, P, P],
            "b200_moe_route": [P, L, P, P, P, P, P, P, P, I, I, I, I, I, P],
            "b200_moe_route_rows": [P, L, P, L, I, I, P, L, P, P, P, P, P, P, P, I, I, I, I, I, I, P],
            "b200_moe_dispatch": [P, L, P, L, P, P, P, P, P, I, I, I, I, I, I, I, P],
            "b200_latent_norm_append": [P, L, P, P, P, L, P, P, I, I, I, I, L, F, I, P, P],
            "b200_latent_gather": [P, P, P, P, P, I, I, I, I, I, I, P, P],
            "b200_latent_rotate": [P, L, P, L, I, I, I, I, P, P, I, P, P, P, P, I, I, I, I, I, I, I, L, F, I, P, P],
            "b200_latent_attn_rows": [P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, I, P, P],
            "b200_latent_decode": [P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, P, P],
            "b200_latent_decode_tc": [P, P, P, P, P, P, P, P, I, I, I, I, I, I, I, I, I, F, P, P],
            "b200_flash_window_fwd": [P, P, P, P, P, P, P, I, I, I, I, P, P, P],
            "b200_retention_chunk": [P, L, P, L, P, P, P, P, P, P, I, I, I, I, I, I, I, I, F, P, P],
            "b200_grouped_prep": [P, L, P, P, P, P, P, P, P, I, I, I, L, P, I, P, P],
            "b200_grouped_prep_whole": [P, L, P, P, P, P, P, P, P, I, I, I, L, P, I, P, P],
            "b200_grouped_rows": [P, P, P, L, P, L, P, I, P, P, P, P, I, I, I, I, I, P, I, P, P],
            "b200_grouped_decode": [P, P, P, L, P, L, P, I, P, P, P, P, P, I, I, I, I, I, P, P, P],
            "b200_grouped_prefill": [P, P, P, L, P, L, P, I, P, P, P, I, I, I, I, I, I, P, P, P],
            "b200_mlstm": [P, L, P, L, P, L, P, L, I, P, P, P, L, P, P, P, P, I, I, I, I, I, I, I, F, F, I, I, P, P],
            "b200_short_conv": [P, P, L, I, I, P, P],
            "b200_short_conv_attend": [P, P, P, P, L, P, P, L, L, I, F, P, I, P, P],
            "b200_group_step": [P, P, P, P, P, P, L, F, I, I, I, I, I, P, P],
            "b200_delta": [P, I, I, P],
            "b200_delta_image_bytes": [],
            "b200_delta_chunk_tokens": [],
            "b200_retention_recurrent": [P, L, P, L, P, P, P, P, P, P, I, I, I, I, I, I, I, I, F, I, P, P],
        }.items():
            fn = getattr(lib, name, None)
            if fn is None:                 # a serving library holds the mixers of one model
                _req(native.lib_path().stem == "_b200_serving", f"symbol {name} is missing from {native.lib_path()}")
                continue
            fn.argtypes, fn.restype = args, ctypes.c_int
        _declared = True
    return lib


def _f32(t) -> int:
    _req(t.dtype in (torch.float32, torch.bfloat16), "activations must be bf16 or fp32")
    return int(t.dtype == torch.float32)


def pitch(n: int) -> int:
    return -(-n // 8) * 8


def rows_buffer(rows: int, n: int, dtype, device):
    """Uninitialised (rows, n) matrix with an 8-element row pitch."""
    return torch.empty((rows, pitch(n)), dtype=dtype, device=device)[:, :n]


def padded_weight(w, dtype, device):
    """(out, in) weight copied to ``device`` with zeros up to an 8-element row pitch."""
    buf = torch.zeros((w.shape[0], pitch(w.shape[1])), dtype=dtype, device=device)
    buf[:, :w.shape[1]] = w.to(device=device, dtype=dtype)
    return buf[:, :w.shape[1]]


# --------------------------------------------------------------------------------- matrix products
ACTS = {None: 0, "gelu": 1, "cap": 2}


def _finish(bias, alpha, act, cap):
    """What becomes of a product's sums, or None if nothing does."""
    _req(act in ACTS and (act != "cap" or cap > 0.0), "unknown activation")
    if bias is None and alpha == 1.0 and act is None:
        return None
    _req(bias is None or (bias.dtype == torch.float32 and bias.is_contiguous()), "a bias is contiguous fp32")
    return native.GemmFinish(_ptr(bias), float(alpha), float(cap), ACTS[act])


def _ref(struct):
    return None if struct is None else ctypes.byref(struct)


def linear(a, w, out=None, accumulate=False, out_dtype=None, bias=None, alpha: float = 1.0, act: str | None = None, cap: float = 0.0):
    """act(alpha * (a (R, K) @ w (N, K)^T + bias)), bias fp32.  ``accumulate`` adds to an fp32 ``out``; act: "gelu" (with erf; stored in
    the activation type), "cap" (cap * tanh(v / cap)) or nothing."""
    if out is None:
        out = rows_buffer(a.shape[0], w.shape[0], out_dtype or a.dtype, a.device)
    if not a.is_cuda:
        r = mixer_torch.finish(a.float() @ w.float().t(), bias, alpha, act, cap)
        out.copy_(out + r if accumulate else r)
        return out
    _req(bias is None or bias.numel() == w.shape[0], "bad bias")
    finish = _finish(bias, alpha, act, cap)
    if a.dtype == torch.bfloat16:
        return native.gemm(a, w, "nt", out=out, accumulate=accumulate, b_stable=True, finish=finish)
    _req(out.dtype == torch.float32 and w.dtype == torch.float32 and a.shape[1] == w.shape[1], "fp32 product of fp32 operands")
    _check(_lib().b200_gemm_f32(_ptr(a), _ptr(w), _ptr(out), a.shape[0], w.shape[0], a.shape[1], a.stride(0), w.stride(0),
                                out.stride(0), int(accumulate), None, 0, 1, 0, 0, _ref(finish), _stream()), "gemm_f32")
    return out


def gemm_rows(a, w, tile_group, n: int, swiglu: bool, act: str | None = None):
    """Every 128-row tile t of a (P, K) times the rows of w that belong to group tile_group[t] (negative: skipped, the
    rows of the result stay undefined).  ``swiglu``: a group has 2 n rows, gate rows first, and the result is
    silu(gate) * up; otherwise n rows and ``act`` of the product."""
    rows = 2 * n if swiglu else n
    if not a.is_cuda:
        return mixer_torch.gemm_rows(a, w, tile_group, rows, n, swiglu, act)
    lib = _lib()
    p, k = a.shape
    _req(tile_group.dtype == torch.int32 and tile_group.is_contiguous() and tile_group.numel() * TILE >= p and p % TILE == 0
         and w.shape[0] % rows == 0 and w.shape[1] == k and not (swiglu and act), "bad grouped product")
    finish = _finish(None, 1.0, act, 0.0)
    if a.dtype == torch.bfloat16:
        out = rows_buffer(p, n, a.dtype, a.device)
        _check(lib.b200_gemm_bf16_grouped(_ptr(a), _ptr(w), _ptr(out), None, p, n, k, a.stride(0), w.stride(0), out.stride(0),
                                          0, _ptr(tile_group), w.shape[0] // rows, rows, 1, 0, 0, int(swiglu), 0, 0, _ref(finish),
                                          _ptr(native.status_word(a.device)), _stream()), "gemm_grouped")
        return out
    out = rows_buffer(p, rows, a.dtype, a.device)
    _check(lib.b200_gemm_f32(_ptr(a), _ptr(w), _ptr(out), p, rows, k, a.stride(0), w.stride(0), out.stride(0), 0,
                             _ptr(tile_group), rows, 1, 0, 0, _ref(finish), _stream()), "gemm_f32")
    if not swiglu:
        return out
    h = rows_buffer(p, n, a.dtype, a.device)
    _check(lib.b200_glu_any(_ptr(out), _ptr(h), p, n, out.stride(0), h.stride(0), 0, 1, _stream()), "glu_any")
    return h


def glu(a, w, n: int, act: str):
    """act(a @ gate^T) * (a @ up^T) for w (2 n, K), gate rows first; act "silu" or "relu"."""
    _req(act in ("silu", "relu") and w.shape[0] == 2 * n and w.shape[1] == a.shape[1], "bad gated product")
    out = rows_buffer(a.shape[0], n, a.dtype, a.device)
    if not a.is_cuda:
        return mixer_torch.glu(a, w, n, act, out)
    lib = _lib()
    m, k = a.shape
    if a.dtype == torch.bfloat16:
        _check(lib.b200_gemm_bf16_grouped(_ptr(a), _ptr(w), _ptr(out), None, m, n, k, a.stride(0), w.stride(0), out.stride(0), 0, None,
                                          0, 2 * n, 1, 0, 0, 2 if act == "relu" else 1, native.EPI_B_STABLE, 0, None,
                                          _ptr(native.status_word(a.device)), _stream()), "gemm_glu")
        return out
    gu = linear(a, w)
    _check(lib.b200_glu_any(_ptr(gu), _ptr(out), m, n, gu.stride(0), out.stride(0), int(act == "relu"), 1, _stream()), "glu_any")
    return out


def gemm_heads(a, w, heads: int, k: int, n: int, out=None, gate=None, a_step: int | None = None, c_step: int | None = None):
    """One product per head, side by side: out[:, h c_step : h c_step + n] = a[:, h a_step : h a_step + k] @ w_h^T, w_h = rows
    [h w.shape[0] / heads, ...) of w (the steps are k and n unless given); ``gate`` multiplies with sigmoid(gate), element by
    element or, with one column per head, head by head."""
    a_step, c_step = a_step or k, c_step or n
    if out is None:
        out = rows_buffer(a.shape[0], heads * n, a.dtype, a.device)
    if not a.is_cuda:
        return mixer_torch.gemm_heads(a, w, heads, k, n, out, gate, a_step, c_step)
    lib = _lib()
    _req(w.shape[0] % heads == 0 and w.shape[1] == k and a.shape[1] >= (heads - 1) * a_step + k
         and out.shape[1] >= (heads - 1) * c_step + n, "bad head product")
    by_head = gate is not None and gate.shape[1] == heads
    _req(gate is None or by_head or (gate.shape[1] >= heads * n and c_step == n), "bad gate")
    if a.dtype == torch.bfloat16:
        _req(k % 8 == 0 and a_step % 8 == 0, "a head's columns must start on a 16-byte boundary")
        epi = (5 if gate is not None else 0) | native.EPI_B_STABLE
        _check(lib.b200_gemm_bf16_grouped(_ptr(a), _ptr(w), _ptr(out), _ptr(gate), a.shape[0], n, k, a.stride(0), w.stride(0),
                                          out.stride(0), 0 if gate is None else gate.stride(0), None, 0, w.shape[0] // heads,
                                          heads, a_step, c_step, 0, epi, int(by_head), None, _ptr(native.status_word(a.device)),
                                          _stream()), "gemm_heads")
        return out
    _check(lib.b200_gemm_f32(_ptr(a), _ptr(w), _ptr(out), a.shape[0], n, k, a.stride(0), w.stride(0), out.stride(0), 0, None,
                             w.shape[0] // heads, heads, a_step, c_step, None, _stream()), "gemm_f32")
    if gate is not None:
        gate_sigmoid_(out, gate)
    return out


def gate_sigmoid_(o, gate):
    """o (R, n) times sigmoid(gate (R, m)), every gate for n / m columns."""
    n, m = o.shape[1], gate.shape[1]
    _req(n % m == 0 and o.shape[0] == gate.shape[0] and o.dtype == gate.dtype, "gate and output must match")
    if not o.is_cuda:
        return o.mul_(torch.sigmoid(gate.float()).repeat_interleave(n // m, 1).to(o.dtype))
    _check(_lib().b200_gate_sigmoid(_ptr(o), _ptr(gate), o.shape[0], n, n // m, o.stride(0), gate.stride(0), _f32(o),
                                    _stream()), "gate_sigmoid")
    return o


# ------------------------------------------------------------------------------- residual and norm
class ExpertOutputs(NamedTuple):
    """What the experts of a layer add to the residual stream: x += scale * (sum_k weight[row, k] * y[pos[row, k]] + sigmoid(sgate[row])
    * s[row]); a choice with pos -2 stands for the experts' input z[row], -1 for none; without ``weight`` all weights are one."""
    y: torch.Tensor
    pos: torch.Tensor                        # (R, top) int32
    scale: float
    weight: torch.Tensor | None = None       # (R, top) fp32
    z: torch.Tensor | None = None
    s: torch.Tensor | None = None
    sgate: torch.Tensor | None = None        # (R,) fp32, any stride


class _NativeOutputs(ctypes.Structure):
    """csrc/mixer_elementwise.cu: ExpertOutputs"""
    _fields_ = [(n, ctypes.c_void_p) for n in ("y", "ypos", "yweight", "z", "s", "sgate")] + \
               [(n, ctypes.c_longlong) for n in ("ld_y", "ld_z", "ld_s", "ld_sgate")] + \
               [("ytop", ctypes.c_int), ("y_rows", ctypes.c_int), ("yscale", ctypes.c_float)]


def _expert_outputs(ex: ExpertOutputs, x, act_dtype):
    rows, d = x.shape
    fits = lambda t, n: t is None or (t.dtype == act_dtype and t.shape == (n, d) and t.stride(1) == 1)
    _req(fits(ex.y, ex.y.shape[0]) and fits(ex.z, rows) and fits(ex.s, rows) and ex.pos.dtype == torch.int32
         and ex.pos.is_contiguous() and ex.pos.shape[0] == rows, "bad expert outputs")
    _req(ex.weight is None or (ex.weight.dtype == torch.float32 and ex.weight.is_contiguous() and ex.weight.shape == ex.pos.shape),
         "bad expert weights")
    _req(ex.sgate is None or (ex.sgate.dtype == torch.float32 and ex.sgate.shape == (rows,)), "bad gate")
    pitch_of = lambda t: 0 if t is None else t.stride(0)
    return _NativeOutputs(_ptr(ex.y), _ptr(ex.pos), _ptr(ex.weight), _ptr(ex.z), _ptr(ex.s), _ptr(ex.sgate), pitch_of(ex.y),
                          pitch_of(ex.z), pitch_of(ex.s), pitch_of(ex.sgate), ex.pos.shape[1], ex.y.shape[0], float(ex.scale))


def residual_norm(x, w=None, eps: float = 0.0, tokens=None, embed=None, row_index=None, pending=None, scatter=None,
                  embed_scale: float = 1.0, w_offset: float = 0.0):
    """One pass over the fp32 residual stream x (R, d):

    * ``tokens`` / ``embed``: x = embed[tokens] * embed_scale first
    * ``pending``: ``ExpertOutputs`` (or its first three fields) to add to x
    * ``w``: h = x / rms(x) * (w + w_offset), returned in w's dtype (no ``w``: only x is updated)
    * ``row_index``: h for these rows of x only, x itself stays as it is
    * ``scatter`` = (pos (R, top), rows): also returns the normed rows at the places the experts read them from

    Returns (h, scattered)."""
    if pending is not None:
        pending = ExpertOutputs(*pending)
    if not x.is_cuda:
        return mixer_torch.residual_norm(x, tokens, embed, row_index, pending, w, eps, scatter, embed_scale, w_offset)
    lib = _lib()
    _req(x.dtype == torch.float32 and x.is_contiguous(), "the residual stream is contiguous fp32")
    d = x.shape[1]
    rows = x.shape[0] if row_index is None else row_index.numel()
    act = w if w is not None else (embed if embed is not None else pending.y)
    h = xg = None
    if w is not None:
        _req(w.numel() == d and w.is_contiguous(), "bad norm weight")
        h = rows_buffer(rows, d, w.dtype, x.device)
    if tokens is not None:
        _req(tokens.dtype == torch.int64 and tokens.numel() == rows and embed.is_contiguous() and embed.shape[1] == d
             and embed.dtype == act.dtype, "bad embedding")
    if row_index is not None:
        _req(row_index.dtype == torch.int64 and row_index.is_contiguous(), "row_index must be int64")
    ex = None if pending is None else _expert_outputs(pending, x, act.dtype)
    gpos, g_rows = scatter if scatter is not None else (None, 0)
    if scatter is not None:
        _req(gpos.dtype == torch.int32 and gpos.is_contiguous() and gpos.shape[0] == rows, "bad expert positions")
        xg = rows_buffer(g_rows, d, w.dtype, x.device)
    _check(lib.b200_residual_norm(
        _ptr(tokens), _ptr(embed), 0 if embed is None else embed.shape[0], float(embed_scale), _ptr(x), _ptr(row_index), _ref(ex),
        _ptr(w), float(w_offset), _ptr(h), 0 if h is None else h.stride(0), float(eps), _ptr(xg), _ptr(gpos),
        0 if gpos is None else gpos.shape[1], g_rows, 0 if xg is None else xg.stride(0), rows, x.shape[0], d, _f32(act),
        _ptr(native.status_word(x.device)), _stream()), "residual_norm")
    return h, xg


def add_normed(x, y=None, w=None, eps: float = 0.0, tokens=None, embed=None):
    """Norm behind a sublayer: x (R, d) fp32 += y / rms(y) * w in place; with ``tokens`` / ``embed`` instead x = embed[tokens].
    Returns x in the activation type, for the next sublayer to read."""
    act = embed if tokens is not None else y
    h = rows_buffer(x.shape[0], x.shape[1], act.dtype, x.device)
    if not x.is_cuda:
        return mixer_torch.add_normed(x, y, w, eps, tokens, embed, h)
    d = x.shape[1]
    _req(x.dtype == torch.float32 and x.is_contiguous(), "the residual stream is contiguous fp32")
    if tokens is not None:
        _req(tokens.dtype == torch.int64 and tokens.numel() == x.shape[0] and embed.is_contiguous() and embed.shape[1] == d, "bad embedding")
    else:
        _req(y.shape == x.shape and y.stride(1) == 1 and w.dtype == y.dtype and w.numel() == d and w.is_contiguous(), "bad sublayer output")
    _check(_lib().b200_add_normed(_ptr(tokens), _ptr(embed), 0 if embed is None else embed.shape[0], _ptr(x), _ptr(y),
                                  0 if y is None else y.stride(0), _ptr(w), _ptr(h), h.stride(0), float(eps), x.shape[0], d, _f32(act),
                                  _ptr(native.status_word(x.device)), _stream()), "add_normed")
    return h


# ------------------------------------------------------------------------------ mixture of experts
def plan_tiles(rows: int, experts: int, top: int, always: int = 0) -> int:
    """Row tiles that ``rows`` tokens can need at most: every expert in use leaves one tile partly empty, and each of the ``always``
    experts receives all rows."""
    return min(experts, rows * top) + rows * top // TILE + always * -(-rows // TILE)


def moe_plan(tokens, slots, tables, experts):
    """Sort the (row, choice) pairs of a step by expert, for several layers at once (each with its own table).
    Returns per layer pos (R, top) int32 and tile_group (tiles,) int32.  Rows with a negative slot are left out."""
    rows = tokens.numel()
    tiles = max(plan_tiles(rows, n, t.shape[1]) for t, n in zip(tables, experts))
    if not tokens.is_cuda:
        return mixer_torch.moe_plan(tokens, slots, tables, experts, tiles)
    lib = _lib()
    _req(tokens.dtype == torch.int64 and slots.dtype == torch.int64 and slots.numel() == rows, "bad plan inputs")
    top = max(t.shape[1] for t in tables)
    pos = torch.empty((len(tables), rows * top), dtype=torch.int32, device=tokens.device)
    group = torch.empty((len(tables), tiles), dtype=torch.int32, device=tokens.device)
    step = lib.b200_moe_plan_layers()
    for a in range(0, len(tables), step):
        part = tables[a:a + step]
        n = len(part)
        for t in part:
            _req(t.dtype == torch.int32 and t.is_contiguous() and t.shape[0] == tables[0].shape[0], "bad expert table")
        ptrs = (ctypes.c_void_p * n)(*[t.data_ptr() for t in part])
        ne = (ctypes.c_int * n)(*experts[a:a + step])
        nt = (ctypes.c_int * n)(*[t.shape[1] for t in part])
        _check(lib.b200_moe_plan(_ptr(tokens), _ptr(slots), rows, tables[0].shape[0], n, ptrs, ne, nt, _ptr(pos[a]),
                                 pos.stride(0), _ptr(group[a]), tiles, _ptr(native.status_word(tokens.device)), _stream()),
               "moe_plan")
    return ([pos[i, :rows * t.shape[1]].view(rows, t.shape[1]) for i, t in enumerate(tables)], [group[i] for i in range(len(tables))])


def moe_route(z, correction, slots, experts: int, top: int, count, always: int = 0, bias=None):
    """Choose experts by score: z (R, outputs) fp32 logits of the experts and, behind them, of identities, plus ``bias``; scores are their
    softmax.  The ``top`` outputs with the largest score + correction (``correction`` None: the largest logits) are chosen and weighted by
    their share of the chosen scores.  ``count``
    (experts,) int32, zero on entry, receives the rows per expert.  ``always``: that many weights sigmoid(z[:, outputs]) more per row
    (z has one more column).  Returns choice (-1 in padding rows) and rank among the expert's rows, (R, top), and weight
    (R, top + always)."""
    rows, outputs = z.shape[0], z.shape[1] - (always > 0)
    _req(0 < top <= outputs and experts <= outputs, "bad router sizes")
    if not z.is_cuda:
        return mixer_torch.moe_route(z, correction, slots, experts, top, count, always, bias)
    _req(z.dtype == torch.float32 and z.stride(1) == 1, "bad logits")
    choice, rank, weight = _route_buffers(rows, outputs, top, always, bias, correction, slots, experts, count)
    _check(_lib().b200_moe_route(_ptr(z), z.stride(0), _ptr(bias), _ptr(correction), _ptr(slots), _ptr(choice), _ptr(rank), _ptr(weight),
                                 _ptr(count), rows, experts, outputs, top, always, _stream()), "moe_route")
    return choice, rank, weight


def _route_buffers(rows, outputs, top, always, bias, correction, slots, experts, count):
    fits = lambda t: t is None or (t.dtype == torch.float32 and t.is_contiguous() and t.numel() == outputs)
    _req(fits(bias) and fits(correction) and count.dtype == torch.int32 and count.is_contiguous()
         and count.numel() == experts and slots.dtype == torch.int64 and slots.numel() == rows, "bad router inputs")
    choice, rank = (torch.empty((rows, top), dtype=torch.int32, device=slots.device) for _ in range(2))
    return choice, rank, torch.empty((rows, top + always), dtype=torch.float32, device=slots.device)


ROUTE_ROWS, ROUTE_BYTES = 256, 32 << 20          # rows, and bytes of the router read once per row, up to which one kernel does it all


def routes_rows(rows: int, w) -> bool:
    """Whether a step of this many rows is routed by ``moe_route_rows``."""
    return w.is_cuda and rows <= ROUTE_ROWS and rows * w.numel() * w.element_size() <= ROUTE_BYTES and 3 * w.shape[0] + w.shape[1] <= 12000


def moe_route_rows(h, w, correction, slots, experts: int, top: int, count, always: int = 0, bias=None):
    """``moe_route`` of the few rows of a decode step with the router's product, z = h w^T in fp32.  Returns z too."""
    (rows, d), columns = h.shape, w.shape[0]
    outputs = columns if correction is None else correction.numel()
    _req(h.is_cuda and h.dtype == w.dtype and h.stride(1) == 1 and w.shape[1] == d and columns >= outputs + (always > 0), "bad router")
    z = torch.empty((rows, columns), dtype=torch.float32, device=h.device)
    choice, rank, weight = _route_buffers(rows, outputs, top, always, bias, correction, slots, experts, count)
    _check(_lib().b200_moe_route_rows(_ptr(h), h.stride(0), _ptr(w), w.stride(0), d, columns, _ptr(z), columns, _ptr(bias), _ptr(correction),
                                      _ptr(slots), _ptr(choice), _ptr(rank), _ptr(weight), _ptr(count), rows, experts, outputs, top, always,
                                      _f32(h), _stream()), "moe_route_rows")
    return z, choice, rank, weight


def moe_dispatch(h, choice, rank, count, always: int = 0):
    """Rows of h sorted by chosen expert into 128-row tiles, then all rows for each of the ``always`` further experts.  Returns them
    (tiles * 128, d), where each choice went, pos (R, top + always) int32 (-2: an identity, -1: none), and the expert of every tile,
    tile_group (tiles,) int32."""
    (rows, top), experts = choice.shape, count.numel()
    tiles = plan_tiles(rows, experts, top, always)
    if not h.is_cuda:
        return mixer_torch.moe_dispatch(h, choice, rank, count, always, tiles)
    _req(h.stride(1) == 1 and h.shape[0] == rows and choice.dtype == torch.int32 and rank.dtype == torch.int32, "bad expert rows")
    xg = rows_buffer(tiles * TILE, h.shape[1], h.dtype, h.device)
    pos = torch.empty((rows, top + always), dtype=torch.int32, device=h.device)
    group = torch.empty((tiles,), dtype=torch.int32, device=h.device)
    _check(_lib().b200_moe_dispatch(_ptr(h), h.stride(0), _ptr(xg), xg.stride(0), _ptr(choice), _ptr(rank), _ptr(count), _ptr(pos),
                                    _ptr(group), rows, experts, top, always, tiles, h.shape[1], h.element_size(), _stream()), "moe_dispatch")
    return xg, pos, group


# -------------------------------------------------------------------------------- latent attention
def latent_norm_append(proj, wq, wkv, eps: float, cache, slots):
    """Norm of both latents in proj (columns [0, q_rank) and [q_rank, q_rank + kv_rank)): returns the query latent and
    writes the key/value latent to its cache slot (negative slot: not written)."""
    qr, kvr = wq.numel(), wkv.numel()
    cq = rows_buffer(proj.shape[0], qr, proj.dtype, proj.device)
    if not proj.is_cuda:
        return mixer_torch.latent_norm_append(proj, wq, wkv, eps, cache, slots, cq)
    _req(cache.is_contiguous() and cache.dtype == proj.dtype and cache.shape[-1] >= kvr and slots.dtype == torch.int64
         and slots.numel() == proj.shape[0], "bad latent cache")
    _check(_lib().b200_latent_norm_append(_ptr(proj), proj.stride(0), _ptr(wq), _ptr(wkv), _ptr(cq), cq.stride(0), _ptr(cache),
                                          _ptr(slots), proj.shape[0], qr, kvr, cache.shape[-1],
                                          cache.shape[0] * cache.shape[1], float(eps), _f32(proj),
                                          _ptr(native.status_word(proj.device)), _stream()), "latent_norm_append")
    return cq


def latent_rotate(q, q_col: int, q_pitch: int, kv, kv_col: int | None, k_col: int | None, wkv, ql, cache, cos_sin, positions, slots,
                  heads: int, kv_rank: int, vwidth: int, rot: int, eps: float):
    """Rotation (interleaved pairs) and append: the heads' rotated query parts are columns q_col + h * q_pitch ... of ``q``; those of
    the first rows go behind the queries in latent space, ``ql`` (rows, heads * width), the others stay in place.  The latent at
    column ``kv_col`` of ``kv`` (None: no latent here) is normed and, with the rotated key part at ``k_col`` (None: none), written to
    its cache slot: latent, then from column ``vwidth`` on the key part."""
    n = 0 if ql is None else ql.shape[0]
    if not q.is_cuda:
        return mixer_torch.latent_rotate(q, q_col, q_pitch, kv, kv_col, k_col, wkv, ql, cache, cos_sin, positions, slots, heads,
                                         kv_rank, vwidth, rot, eps)
    width = cache.shape[-1]
    _req(cache.is_contiguous() and cache.dtype == q.dtype and slots.dtype == torch.int64 and slots.numel() == q.shape[0]
         and positions.dtype == torch.int32 and q.stride(1) == 1 and kv.stride(1) == 1 and kv.dtype == q.dtype
         and kv.shape[0] == q.shape[0], "bad latent cache or rows")
    _req(cos_sin.dtype == torch.float32 and cos_sin.is_contiguous() and cos_sin.shape[2] == rot // 2, "bad rotary table")
    _req(ql is None or (ql.is_contiguous() and ql.dtype == q.dtype and ql.shape[1] == heads * width), "bad latent queries")
    _check(_lib().b200_latent_rotate(
        _ptr(q), q.stride(0), _ptr(kv), kv.stride(0), q_col, q_pitch, -1 if kv_col is None else kv_col, -1 if k_col is None else k_col, _ptr(wkv), _ptr(ql),
        n, _ptr(cache), _ptr(cos_sin), _ptr(positions), _ptr(slots), q.shape[0], heads, kv_rank, vwidth, width, rot, cos_sin.shape[1],
        cache.shape[0] * cache.shape[1], float(eps), _f32(q), _ptr(native.status_word(q.device)), _stream()), "latent_rotate")


def latent_attention_rows(q, cache, row_seq, positions, slots, tables, heads: int, window: int, scale: float, vwidth: int | None = None):
    """q (R, heads * width) in latent space against the paged latents; every row has its own position and line of
    ``tables`` (``row_seq`` None: line i for row i).  window 0 = none.  Returns (R, heads * vwidth): what is summed up are the first
    ``vwidth`` columns of a cached vector (all of them unless given)."""
    vwidth = vwidth or cache.shape[-1]
    if not q.is_cuda:
        return mixer_torch.latent_attention(q, cache, row_seq, positions, slots, tables, heads, window, scale, vwidth)
    _req(q.is_contiguous() and cache.is_contiguous() and q.dtype == cache.dtype and q.shape[1] == heads * cache.shape[-1],
         "bad latent queries")
    _req(tables.dtype == torch.int32 and tables.is_contiguous() and positions.dtype == torch.int32, "bad tables")
    out = torch.empty((q.shape[0], heads * vwidth), dtype=q.dtype, device=q.device)
    _check(_lib().b200_latent_attn_rows(_ptr(q), _ptr(cache), _ptr(out), _ptr(row_seq), _ptr(positions), _ptr(slots),
                                        _ptr(tables), tables.shape[0], q.shape[0], heads, cache.shape[-1], vwidth, tables.shape[1],
                                        cache.shape[1], cache.shape[0], window, float(scale), _f32(q),
                                        _ptr(native.status_word(q.device)), _stream()), "latent_attn_rows")
    return out


DECODE_MAX_WIDTH, DECODE_MAX_KEY = 512, 576      # what the tensor-core decode kernels sum up, and score, of a cached vector
DECODE_TILE = 32


def latent_splits(rows: int, heads: int, keys: int, sms: int = 148) -> int:
    """Splits of the window per row of a decode step, by a cost in tiles: a CTA starts up for about two tiles, two CTAs that
    share an SM (up to 16 heads; with more there is one) take 1.7 times as long as one, a merge costs about two tiles."""
    groups = rows * (1 if heads <= 16 else -(-heads // 32))
    best, best_cost = 1, None
    for n in range(1, max(1, min(32, keys // (2 * DECODE_TILE))) + 1):
        per_sm = -(-groups * n // sms)
        load = per_sm if heads > 16 else per_sm // 2 * 1.7 + per_sm % 2
        cost = load * (-(-keys // (n * DECODE_TILE)) + 2) + (2 if n > 1 else 0)
        if best_cost is None or cost < best_cost:
            best, best_cost = n, cost
    return best


def latent_splits_tc(rows: int, keys: int, sms: int = 148) -> int:
    """The same for the tcgen05 kernel: one CTA per SM, tiles of 128 tokens (one more for the page border the window starts
    behind), a start-up worth about one and a half tiles and a merge worth about one."""
    best, best_cost = 1, None
    for n in range(1, max(1, min(16, keys // 256)) + 1):
        cost = -(-rows * n // sms) * (-(-(keys // 128 + 1) // n) + 1.5) + (1 if n > 1 else 0)
        if best_cost is None or cost < best_cost:
            best, best_cost = n, cost
    return best


def latent_decode(q, cache, positions, slots, tables, heads: int, window: int, scale: float, splits: int = 0, kernel: str = "auto",
                  vwidth: int | None = None):
    """``latent_attention_rows`` for one query row per request: line i of ``tables`` belongs to row i.  ``kernel``: "tcgen05"
    (vwidths that are multiples of 128, up to 64 columns behind them, up to 64 heads, pages that divide 128), "mma" (any width up to
    ``DECODE_MAX_KEY``), "rows"; "auto" takes the first that fits, and "mma" for small batches, whose CTAs it spreads over the SMs
    with shorter chains."""
    width, page = cache.shape[-1], cache.shape[1]
    vwidth = vwidth or width
    if kernel == "auto":
        fits = q.is_cuda and q.dtype == torch.bfloat16 and vwidth <= DECODE_MAX_WIDTH and width <= DECODE_MAX_KEY
        tc = (fits and vwidth % 128 == 0 and width <= vwidth + 64 and heads <= 64 and page >= 8 and 128 % page == 0
              and q.shape[0] * max(heads, 16) >= 1024)
        kernel = "tcgen05" if tc else ("mma" if fits else "rows")
    if kernel == "rows":
        return latent_attention_rows(q, cache, None, positions, slots, tables, heads, window, scale, vwidth)
    rows = q.shape[0]
    _req(q.is_contiguous() and cache.is_contiguous() and q.shape[1] == heads * width and tables.shape[0] >= rows, "bad latent queries")
    _req(q.dtype == torch.bfloat16 and cache.dtype == q.dtype, "bf16 queries and latents")
    _req(tables.dtype == torch.int32 and tables.is_contiguous() and positions.dtype == torch.int32, "bad tables")
    keys = tables.shape[1] * page
    keys = min(window, keys) if window > 0 else keys
    if kernel == "tcgen05":
        fn, splits = _lib().b200_latent_decode_tc, splits or latent_splits_tc(rows, keys)
    else:
        fn, splits = _lib().b200_latent_decode, splits or latent_splits(rows, heads, keys)
    out = torch.empty((rows, heads * vwidth), dtype=q.dtype, device=q.device)
    part = torch.empty(rows * heads * splits * (vwidth + 2) if splits > 1 else 0, dtype=torch.float32, device=q.device)
    ml = part[rows * heads * splits * vwidth:]
    _check(fn(_ptr(q), _ptr(cache), _ptr(out), _ptr(part), _ptr(ml), _ptr(positions), _ptr(slots), _ptr(tables), rows, heads, width,
              vwidth, tables.shape[1], page, cache.shape[0], window, splits, float(scale), _ptr(native.status_word(q.device)), _stream()),
           "latent_decode" if splits > 1 else "latent_decode_one")
    return out


def latent_gather(cache, cu_k, first_k, tables, total: int):
    """Cached latents of the keys a step's portions can see, packed (total, width): rows cu_k[b] .. of portion b start at
    position first_k[b]."""
    width = cache.shape[-1]
    out = torch.empty((total, width), dtype=cache.dtype, device=cache.device)
    _req(cache.dtype == torch.bfloat16 and cache.is_contiguous() and tables.dtype == torch.int32 and tables.is_contiguous(), "bad cache")
    _check(_lib().b200_latent_gather(_ptr(cache), _ptr(out), _ptr(cu_k), _ptr(first_k), _ptr(tables), cu_k.numel() - 1, total,
                                     tables.shape[1], cache.shape[1], cache.shape[0], width,
                                     _ptr(native.status_word(cache.device)), _stream()), "latent_gather")
    return out


class _WindowShape(ctypes.Structure):
    """csrc/flash_attn_fwd.cu: FlashWindowShape"""
    _fields_ = [(n, ctypes.c_longlong) for n in ("ld_q", "ld_kv", "ld_kr", "ld_o", "ld_gate")] + \
               [(n, ctypes.c_int) for n in ("q_cols", "kv_cols", "kr_cols", "heads", "dim", "vdim", "q_step", "k_step", "v_step", "v_off",
                                            "rot", "qr_col", "qr_step", "kr_col", "window", "head_gate")] + [("scale", ctypes.c_float)]


def window_attention(q, kv, cu_q, cu_k, max_q: int, heads: int, dim: int, vdim: int, window: int, scale: float, out, gate=None,
                     steps=None, rot=None):
    """Softmax attention of packed portions under a sliding window (0 = none) on the tensor cores: a head's queries are ``dim`` columns of
    q (Rq, ...), its keys and values ``dim`` and ``vdim`` columns of kv (Rk, ...), up to 128 each; the queries of a portion are the
    last positions of its keys.  ``steps`` = (q_step, k_step, v_step, v_off): head h starts at columns h q_step, h k_step,
    v_off + h v_step (default: heads of ``dim`` columns side by side, all keys before all values); columns from ``dim`` up to the next
    multiple of 16 must be finite, and zero in q or kv.  ``rot`` = (kr (Rk, ...), dims, qr_col, qr_step, kr_col): the scores gain
    rotated parts, ``dims`` (up to 64) columns of q at qr_col + h qr_step and of kr, for all heads, at kr_col.
    out (Rq, heads * vdim), times sigmoid(gate), element by element or with a column per head."""
    q_step, k_step, v_step, v_off = steps or (dim, dim, dim, heads * dim)
    kr, dims, qr_col, qr_step, kr_col = rot or (None, 0, 0, 0, 0)
    _req(q.dtype == torch.bfloat16 and kv.dtype == torch.bfloat16 and q.stride(1) == 1 and kv.stride(1) == 1, "bf16 queries and keys")
    _req(q.shape[1] >= (heads - 1) * q_step + dim and kv.shape[1] >= max((heads - 1) * k_step + dim, v_off + (heads - 1) * v_step + vdim)
         and out.shape == (q.shape[0], heads * vdim), "bad shapes")
    _req(kr is None or (kr.dtype == torch.bfloat16 and kr.stride(1) == 1 and kr.shape[0] == kv.shape[0] and kr.shape[1] >= kr_col + dims
                        and q.shape[1] >= qr_col + (heads - 1) * qr_step + dims), "bad rotated parts")
    _req(gate is None or gate.shape in ((q.shape[0], heads), tuple(out.shape)), "bad gate")
    _req(cu_q.dtype == torch.int32 and cu_k.dtype == torch.int32 and cu_q.numel() == cu_k.numel(), "bad row offsets")
    by_head = gate is not None and gate.shape[1] == heads
    shape = _WindowShape(q.stride(0), kv.stride(0), 0 if kr is None else kr.stride(0), out.stride(0), 0 if gate is None else gate.stride(0),
                         q.shape[1], kv.shape[1], 0 if kr is None else kr.shape[1], heads, dim, vdim, q_step, k_step, v_step, v_off,
                         dims, qr_col, qr_step, kr_col, window, int(by_head), float(scale))
    _check(_lib().b200_flash_window_fwd(
        _ptr(q), _ptr(kv), _ptr(kr), _ptr(out), _ptr(gate), _ptr(cu_q), _ptr(cu_k), cu_q.numel() - 1, max_q, q.shape[0], kv.shape[0],
        ctypes.byref(shape), _ptr(native.status_word(q.device)), _stream()), "flash_window_fwd")
    return out


# --------------------------------------------------------------------------------------- retention
CHUNK = 128                      # tokens per chunk of the tensor-core prompt kernel


def retention_powers(decay, device):
    """decay^m for m = 0 .. CHUNK per head, (heads, CHUNK + 1) fp32 rounded from double, for ``retention_chunked``; None when
    a head forgets so fast that a chunk's powers would leave the range the kernel's scaled rows can have."""
    d = torch.tensor([float(x) for x in decay], dtype=torch.float64)
    if len(d) == 0 or float(d.min()) < 2.0 ** (-40.0 / (CHUNK - 1)) or float(d.max()) > 2.0 ** (40.0 / (CHUNK - 1)):
        return None
    return (d[:, None] ** torch.arange(CHUNK + 1, dtype=torch.float64)).float().contiguous().to(device)


def chunkable(dtype, dim: int, vdim: int, rot: int) -> bool:
    return dtype == torch.bfloat16 and dim % 8 == 0 and vdim % 8 == 0 and dim <= 128 and vdim <= 128 and rot % 16 == 0


def retention_chunked(proj, state, state_slots, cu, positions, cos_sin, powers, heads: int, dim: int, vdim: int, rot: int,
                      eps: float, y):
    """``retention`` for portions of prompts on the tensor cores (bf16 projections, fp32 state and accumulation)."""
    _req(chunkable(proj.dtype, dim, vdim, rot) and proj.is_cuda, "sizes the chunked kernel does not take")
    _req(state.dtype == torch.float32 and state.is_contiguous() and state.shape[1:] == (heads, dim, vdim), "bad state")
    _req(state_slots.dtype == torch.int32 and positions.dtype == torch.int32 and cu.dtype == torch.int32
         and cu.numel() == state_slots.numel() + 1 and powers.shape == (heads, CHUNK + 1), "bad inputs")
    _req(proj.shape[1] == 2 * heads * (dim + vdim) and y.shape == (proj.shape[0], heads * vdim) and y.dtype == proj.dtype, "bad shapes")
    _check(_lib().b200_retention_chunk(
        _ptr(proj), proj.stride(0), _ptr(y), y.stride(0), _ptr(state), _ptr(state_slots), _ptr(cu), _ptr(positions),
        _ptr(cos_sin), _ptr(powers), state_slots.numel(), proj.shape[0], heads, dim, vdim, rot,
        0 if rot == 0 else cos_sin.shape[1], state.shape[0], float(eps), _ptr(native.status_word(proj.device)), _stream()),
        "retention_chunk")
    return y


def retention(proj, state, state_slots, cu, spans, positions, cos_sin, decay, heads: int, dim: int, vdim: int, rot: int,
              eps: float, y):
    """Retention over the rows of ``proj`` (q | k | v | gate).  ``cu`` (sequences + 1, int32) delimits the sequences, None
    = one row each; ``spans`` says the same on the host.  The states are read and left in their slots; y (R, heads * vdim)
    receives the normalised, gated heads."""
    if not proj.is_cuda:
        return mixer_torch.retention(proj, state, state_slots, spans, positions, cos_sin, decay, heads, dim, vdim, rot, eps, y)
    seqs = state_slots.numel()
    _req(state.dtype == torch.float32 and state.is_contiguous() and state.shape[1:] == (heads, dim, vdim), "bad state")
    _req(state_slots.dtype == torch.int32 and positions.dtype == torch.int32 and decay.dtype == torch.float32, "bad inputs")
    _req(rot == 0 or (cos_sin.dtype == torch.float32 and cos_sin.is_contiguous() and cos_sin.shape[2] == rot // 2), "bad rotary table")
    _req(proj.shape[1] == 2 * heads * (dim + vdim) and y.shape == (proj.shape[0], heads * vdim) and y.dtype == proj.dtype, "bad shapes")
    _check(_lib().b200_retention_recurrent(
        _ptr(proj), proj.stride(0), _ptr(y), y.stride(0), _ptr(state), _ptr(state_slots), _ptr(cu), _ptr(positions),
        _ptr(cos_sin), _ptr(decay), seqs, proj.shape[0], heads, dim, vdim, rot, 0 if rot == 0 else cos_sin.shape[1],
        state.shape[0], float(eps), _f32(proj), _ptr(native.status_word(proj.device)), _stream()), "retention")
    return y


# --------------------------------------------------------------------------------- matrix memory (mLSTM)
def mlstm_state(dim: int, vdim: int) -> int:
    """Floats of one head's state: S (dim, vdim) | n (dim) | m, rounded up to 16 bytes."""
    return -(-(dim * vdim + dim + 1) // 4) * 4


def mlstm_chunkable(dtype, dim: int, vdim: int) -> bool:
    return dtype == torch.bfloat16 and dim % 8 == 0 and vdim % 8 == 0 and dim <= 128 and vdim <= 128


def mlstm_steps(dim: int, vdim: int) -> bool:
    """Whether a decode step of these sizes runs on the one-pass kernel, which also takes the gates' products itself."""
    groups = vdim // 4
    return vdim % 4 == 0 and dim % 2 == 0 and 0 < groups <= 256 and -(-dim // max(1, 256 // groups)) <= 16


def mlstm(proj, gates, gate_bias, weight, state, state_slots, cu, spans, positions, heads: int, dim: int, vdim: int, cap: float,
          eps: float, y, chunked: bool = False):
    """Matrix memory over the rows of ``proj`` (q | k | v | output gate) with the gates' pre-activations ``gates`` (input | forget,
    fp32, without bias; or, for a decode step of ``mlstm_steps`` sizes, the pair (input rows h, the gates' weights)).  ``cu`` (sequences + 1, int32) delimits the sequences, None = one row each; ``spans`` says the same on
    the host.  The states are read and left in their slots; y (R, heads * vdim) receives the normed, weighted, gated heads.
    ``chunked``: the tensor-core kernel for portions of prompts (``mlstm_chunkable`` sizes)."""
    h = w_gates = None
    if isinstance(gates, tuple):
        h, w_gates = gates
        gates = None if proj.is_cuda else h.float() @ w_gates.float().t()
    if not proj.is_cuda:
        return mixer_torch.mlstm(proj, gates, gate_bias, weight, state, state_slots, spans, positions, heads, dim, vdim, cap, eps, y)
    seqs = state_slots.numel()
    _req(state.dtype == torch.float32 and state.is_contiguous() and state.shape[1:] == (heads, mlstm_state(dim, vdim)), "bad state")
    _req(state_slots.dtype == torch.int32 and positions.dtype == torch.int32 and gate_bias.dtype == torch.float32
         and gate_bias.numel() == 2 * heads, "bad inputs")
    if gates is None:
        _req(h.dtype == proj.dtype and w_gates.dtype == proj.dtype and h.shape[0] == proj.shape[0] and h.stride(1) == 1
             and w_gates.shape == (2 * heads, h.shape[1]) and cu is None and mlstm_steps(dim, vdim), "bad inputs of the gates")
    else:
        _req(gates.dtype == torch.float32 and gates.shape == (proj.shape[0], 2 * heads), "bad gates")
    _req(proj.shape[1] == 2 * heads * (dim + vdim) and y.shape == (proj.shape[0], heads * vdim) and y.dtype == proj.dtype
         and weight.dtype == proj.dtype and weight.numel() == heads * vdim, "bad shapes")
    _req(cu is None or (cu.dtype == torch.int32 and cu.numel() == seqs + 1), "bad row offsets")
    _req(not chunked or (mlstm_chunkable(proj.dtype, dim, vdim) and cu is not None), "sizes the chunked kernel does not take")
    _check(_lib().b200_mlstm(
        _ptr(proj), proj.stride(0), _ptr(gates), 0 if gates is None else gates.stride(0), _ptr(h), 0 if h is None else h.stride(0),
        _ptr(w_gates), 0 if h is None else w_gates.stride(0), 0 if h is None else h.shape[1], _ptr(gate_bias), _ptr(weight), _ptr(y), y.stride(0), _ptr(state),
        _ptr(state_slots), _ptr(cu), _ptr(positions), seqs, proj.shape[0], heads, dim, vdim, state.shape[2], state.shape[0],
        float(cap), float(eps), _f32(proj), int(chunked), _ptr(native.status_word(proj.device)), _stream()),
        "mlstm_chunk" if chunked else "mlstm")
    return y


# ------------------------------------------------------------------------------- grouped attention
@dataclass
class AttentionShape:
    """Sizes and constants of one grouped attention (``models.mixers.GroupedAttention``); ``bias`` (heads, n) fp32 holds the bias
    per distance, distances from n - 1 on read its last column; ``slopes`` (heads,) fp32 takes slope * distance off instead.  ``chunked``:
    position i sees j <= i in the same chunk of ``window`` positions.  ``head_gate``: the output gate has a column per head.  ``softcap`` 0: scores are not capped; ``sink`` (heads,) fp32 or None;
    ``whole_norm``: one norm over all queries (and keys) of a token instead of one per head."""
    heads: int
    kv_heads: int
    maps: int
    dim: int
    vdim: int
    rot: int
    scale: float
    window: int
    eps: float
    difference: float = 0.0
    out_scale: float = 1.0
    bias: torch.Tensor | None = None
    keep: int = 0
    softcap: float = 0.0
    sink: torch.Tensor | None = None
    whole_norm: bool = False
    slopes: torch.Tensor | None = None
    chunked: bool = False
    head_gate: bool = False

    @property
    def q_pitch(self) -> int:
        return pitch(self.dim) if self.dim > 128 else (64 if self.dim <= 64 else 128)

    @property
    def k_pitch(self) -> int:
        return pitch(self.dim)

    @property
    def v_pitch(self) -> int:
        return pitch(self.vdim)

    @property
    def cache_width(self) -> int:
        """Elements a token takes in the cache: the keys of all heads and maps, then the values."""
        return self.kv_heads * (self.maps * self.k_pitch + self.v_pitch)


class _NativeShape(ctypes.Structure):
    """csrc/grouped_attention.cuh: GroupedShape"""
    _fields_ = [(n, ctypes.c_int) for n in ("heads", "kv_heads", "maps", "dim", "vdim", "qp", "kp", "vp", "window", "keep")] + \
               [(n, ctypes.c_float) for n in ("scale", "eps", "difference", "out_scale", "softcap")] + \
               [("sink", ctypes.c_void_p), ("slopes", ctypes.c_void_p), ("chunked", ctypes.c_int), ("head_gate", ctypes.c_int)]


def _native_shape(s: AttentionShape):
    got = s.__dict__.get("_native")
    if got is None:
        got = s.__dict__["_native"] = _NativeShape(s.heads, s.kv_heads, s.maps, s.dim, s.vdim, s.q_pitch, s.k_pitch, s.v_pitch,
                                                   s.window, s.keep, s.scale, s.eps, s.difference, s.out_scale, s.softcap,
                                                   _ptr(s.sink), _ptr(s.slopes), int(s.chunked), int(s.head_gate))
    return ctypes.byref(got)


BIAS_MAX = 6000                  # entries of a distance table that fit the portions kernel's shared memory


def attention_tiles(s: AttentionShape, dtype) -> bool:
    """Whether portions of prompts run on the tensor-core kernel."""
    if dtype != torch.bfloat16 or s.dim > 128 or s.vdim > 128:
        return False
    if s.softcap > 0 and (s.bias is not None or s.maps != 1):
        return False
    return s.scale > 0 if s.bias is None else s.bias.shape[1] <= BIAS_MAX


def attention_pages(page_size: int) -> bool:
    return page_size >= 8 and 128 % page_size == 0


def attention_prepare(proj, s: AttentionShape, wq, wk, cos_sin, positions, slots, cache):
    """Queries of ``proj`` (q | k | v | ..., or q | ... without ``wk``) normed (per head, or over all of them) and rotated, (R, heads * maps * q_pitch) with zeros
    behind every head; keys, likewise, and values go to their cache slots (negative slot: not written)."""
    q = torch.empty((proj.shape[0], s.heads * s.maps * s.q_pitch), dtype=proj.dtype, device=proj.device)
    if not proj.is_cuda:
        return mixer_torch.attention_prepare(proj, s, wq, wk, cos_sin, positions, slots, cache, q)
    _req(cache.is_contiguous() and cache.dtype == proj.dtype and cache.shape[-1] == s.cache_width and slots.dtype == torch.int64
         and slots.numel() == proj.shape[0] and positions.dtype == torch.int32 and wq.dtype == proj.dtype, "bad cache or rows")
    _req(s.rot == 0 or (cos_sin.dtype == torch.float32 and cos_sin.is_contiguous() and cos_sin.shape[2] == s.rot // 2), "bad rotary table")
    norm = lambda n: s.dim if not s.whole_norm else n * s.dim
    _req(wq.numel() == norm(s.heads) and wq.is_contiguous() and (wk is None or (wk.numel() == norm(s.kv_heads) and wk.is_contiguous())),
         "bad norm weights")
    fn = _lib().b200_grouped_prep_whole if s.whole_norm else _lib().b200_grouped_prep
    _check(fn(_ptr(proj), proj.stride(0), _ptr(q), _ptr(cache), _ptr(wq), _ptr(wk), _ptr(cos_sin),
                                    _ptr(positions), _ptr(slots), proj.shape[0], s.rot, cos_sin.shape[1] if s.rot else 0,
                                    cache.shape[0] * cache.shape[1], _native_shape(s), _f32(proj),
                                    _ptr(native.status_word(proj.device)), _stream()), "grouped_prep")
    return q


def _attention_args(q, s, cache, positions, tables, out, gate):
    _req(q.is_contiguous() and q.shape[1] == s.heads * s.maps * s.q_pitch and cache.is_contiguous() and cache.dtype == q.dtype
         and cache.shape[-1] == s.cache_width, "bad queries or cache")
    _req(tables.dtype == torch.int32 and tables.is_contiguous() and positions.dtype == torch.int32, "bad tables")
    _req(out.shape == (q.shape[0], s.heads * s.vdim) and out.dtype == q.dtype and out.stride(1) == 1, "bad output")
    _req(gate is None or (gate.shape == (out.shape[0], s.heads if s.head_gate else out.shape[1]) and gate.dtype == q.dtype and gate.stride(1) == 1), "bad gate")
    return (_ptr(q), _ptr(cache), _ptr(out), out.stride(0), _ptr(gate), 0 if gate is None else gate.stride(0), _ptr(s.bias),
            0 if s.bias is None else s.bias.shape[1])


def attention_rows(q, s: AttentionShape, cache, row_seq, positions, slots, tables, out, gate=None):
    """The general form: every row of q has its own position and line of ``tables`` (``row_seq`` None: line i for row i)."""
    if not q.is_cuda:
        return mixer_torch.attention_rows(q, s, cache, row_seq, positions, slots, tables, out, gate)
    args = _attention_args(q, s, cache, positions, tables, out, gate)
    _check(_lib().b200_grouped_rows(*args, _ptr(row_seq), _ptr(positions), _ptr(slots), _ptr(tables), tables.shape[0], q.shape[0],
                                    tables.shape[1], cache.shape[1], cache.shape[0], _native_shape(s), _f32(q),
                                    _ptr(native.status_word(q.device)), _stream()), "grouped_rows")
    return out


def attention_splits(s: AttentionShape, rows: int, keys: int, sms: int = 148) -> int:
    """Splits of the window per row of a decode step: CTAs of four warps that walk 16 tokens at a time, two CTAs to an SM; a start-up
    is worth about three steps, a merge about two."""
    groups = rows * s.kv_heads * -(-(s.heads // s.kv_heads) // (16 // s.maps))
    best, best_cost = 1, None
    for n in range(1, max(1, min(32, keys // 128)) + 1):
        cost = -(-groups * n // (2 * sms)) * (-(-keys // (n * 64)) + 3) + (2 if n > 1 else 0)
        if best_cost is None or cost < best_cost:
            best, best_cost = n, cost
    return best


def attention_decode(q, s: AttentionShape, cache, positions, slots, tables, out, gate=None, splits: int = 0):
    """``attention_rows`` for one query row per request: line i of ``tables`` belongs to row i."""
    fits = q.is_cuda and q.dtype == torch.bfloat16 and s.maps * s.k_pitch <= 256 and s.v_pitch <= 128
    if not fits:
        return attention_rows(q, s, cache, None, positions, slots, tables, out, gate)
    rows, keys = q.shape[0], min(s.window + s.keep, tables.shape[1] * cache.shape[1])
    _req(tables.shape[0] >= rows, "bad tables")
    args = _attention_args(q, s, cache, positions, tables, out, gate)
    splits = splits or attention_splits(s, rows, keys)
    n = rows * s.heads * s.maps * splits
    part = torch.empty(n * (s.vdim + 2) if splits > 1 else 0, dtype=torch.float32, device=q.device)
    _check(_lib().b200_grouped_decode(*args, _ptr(part), _ptr(part[n * s.vdim:]), _ptr(positions), _ptr(slots), _ptr(tables), rows,
                                      tables.shape[1], cache.shape[1], cache.shape[0], splits, _native_shape(s),
                                      _ptr(native.status_word(q.device)), _stream()),
           "grouped_decode" if splits > 1 else "grouped_decode_one")
    return out


def attention_portions(q, s: AttentionShape, cache, positions, cu, max_q: int, tables, out, gate=None):
    """Portions of prompts on the tensor cores: rows cu[b] .. cu[b + 1] - 1 of q belong to portion b, line b of ``tables`` to it; its
    keys and values are in the cache already."""
    _req(attention_tiles(s, q.dtype) and attention_pages(cache.shape[1]) and q.is_cuda, "sizes the portions kernel does not take")
    _req(cu.dtype == torch.int32 and tables.shape[0] >= cu.numel() - 1, "bad row offsets")
    args = _attention_args(q, s, cache, positions, tables, out, gate)
    _check(_lib().b200_grouped_prefill(*args, _ptr(cu), _ptr(positions), _ptr(tables), cu.numel() - 1, max_q, q.shape[0],
                                       tables.shape[1], cache.shape[1], cache.shape[0], _native_shape(s),
                                       _ptr(native.status_word(q.device)), _stream()), "grouped_prefill")
    return out


# --------------------------------------------------------------------------------------- short convolution
class _ConvInput(ctypes.Structure):
    """csrc/short_conv.cu: ConvInput"""
    _fields_ = [(n, ctypes.c_void_p) for n in ("u", "w", "ring", "state_slots", "row_seq", "cu", "positions")] + \
               [("ld_u", ctypes.c_longlong)] + [(n, ctypes.c_int) for n in ("seq0", "seqs", "rows", "channels", "taps", "num_slots")]


class StepRows(NamedTuple):
    """A part of a step's rows: single rows (``cu`` None) or portions."""
    positions: torch.Tensor                  # (R,) int32
    slots: torch.Tensor                      # (R,) int64 cache slots
    state_slots: torch.Tensor                # (sequences,) int32
    row_seq: torch.Tensor                    # (R,) int32, the first sequence is ``seq0``
    seq0: int
    cu: torch.Tensor | None                  # (sequences + 1,) int32
    spans: list                              # the same on the host: (first row, one past the last)


def step_parts(batch):
    """(rows, StepRows) of a step's single rows and of its portions, those that it has."""
    n, rows = batch.n_single, batch.n_rows
    out = []
    if n:
        one = slice(0, n)
        out.append((one, StepRows(batch.positions[one], batch.slots[one], batch.state_slots[one], batch.row_seq[one], 0, None,
                                  [(i, i + 1) for i in range(n)])))
    if rows > n:
        rest = slice(n, rows)
        out.append((rest, StepRows(batch.positions[rest], batch.slots[rest], batch.state_slots[n:], batch.row_seq[rest], n, batch.cu,
                                   batch.spans)))
    return out


def _conv_input(u, w, ring, at: StepRows):
    taps, channels = w.shape
    _req(u.shape[1] == channels and u.stride(1) == 1 and w.is_contiguous() and w.dtype == u.dtype, "bad convolution")
    _req(ring.dtype == u.dtype and ring.is_contiguous() and ring.shape[1:] == (taps, channels), "bad ring")
    _req(at.positions.dtype == torch.int32 and at.positions.numel() == u.shape[0] and at.state_slots.dtype == torch.int32
         and at.row_seq.dtype == torch.int32 and at.row_seq.numel() == u.shape[0], "bad rows")
    _req(at.cu is None or (at.cu.dtype == torch.int32 and at.cu.numel() == at.state_slots.numel() + 1), "bad row offsets")
    single = at.cu is None
    return _ConvInput(_ptr(u), _ptr(w), _ptr(ring), _ptr(at.state_slots), None if single else _ptr(at.row_seq), _ptr(at.cu),
                      _ptr(at.positions), u.stride(0), at.seq0, at.state_slots.numel(), u.shape[0], channels, taps, ring.shape[0])


def short_conv(u, w, ring, at: StepRows, y, silu: bool = False):
    """Causal convolution over time: y_t = sum_j w[j] u_(t - taps + 1 + j) per channel, zeros in front of a sequence; w (taps, channels).
    ``ring`` (slots, taps, channels) holds what earlier steps brought and receives what later ones need."""
    if not u.is_cuda:
        return y.copy_(mixer_torch.short_conv(u, w, ring, at, silu))
    _req(y.shape == u.shape and y.dtype == u.dtype and y.stride(1) == 1, "bad output")
    arg = _conv_input(u, w, ring, at)
    _check(_lib().b200_short_conv(ctypes.byref(arg), _ptr(y), y.stride(0), int(silu), _f32(u), _ptr(native.status_word(u.device)), _stream()),
           "short_conv")
    return y


def conv_attend(u, w, ring, at: StepRows, s: AttentionShape, temp, cache, first=None, mix: float = 0.0):
    """The short convolution of q | k | v: returns the queries, times ``temp`` (heads,) fp32, (R, heads * q_pitch) with zeros behind every head;
    keys and values go to their cache slots (negative slot: not written).  ``first``: another layer's cache; its values of the same
    token join with weight ``mix``, v <- (1 - mix) v + mix v_first."""
    q = torch.empty((u.shape[0], s.heads * s.q_pitch), dtype=u.dtype, device=u.device)
    if not u.is_cuda:
        return mixer_torch.conv_attend(u, w, ring, at, s, temp, cache, first, mix, q)
    arg = _conv_input(u, w, ring, at)
    _req(cache.is_contiguous() and cache.dtype == u.dtype and cache.shape[-1] == s.cache_width and at.slots.dtype == torch.int64
         and at.slots.numel() == u.shape[0] and temp.dtype == torch.float32 and temp.numel() == s.heads, "bad cache or rows")
    width = 0 if first is None else first.shape[-1]
    _req(first is None or (first.is_contiguous() and first.dtype == u.dtype and first.shape[:2] == cache.shape[:2]
                           and width >= s.kv_heads * s.v_pitch), "bad cache of the first values")
    _check(_lib().b200_short_conv_attend(
        ctypes.byref(arg), _ptr(q), _ptr(cache), _ptr(at.slots), cache.shape[0] * cache.shape[1], _ptr(temp), _ptr(first), width,
        width - s.kv_heads * s.v_pitch, s.v_pitch, float(mix), _native_shape(s), _f32(u), _ptr(native.status_word(u.device)), _stream()),
        "short_conv_attend")
    return q


# ------------------------------------------------------------------------------------------ gated delta rule
class _DeltaArgs(ctypes.Structure):
    """csrc/delta.cu: DeltaArgs"""
    _fields_ = [(n, ctypes.c_void_p) for n in ("c", "gate", "ab", "h", "w_ab", "decay", "dt", "weight", "filter", "ring", "y", "state", "image",
                                               "state_slots", "cu", "positions", "chunk_cu", "status")] + \
               [(n, ctypes.c_longlong) for n in ("ld_c", "ld_gate", "ld_ab", "ld_h", "ld_w", "ld_y")] + \
               [(n, ctypes.c_int) for n in ("width", "taps", "seqs", "rows", "heads", "kv_heads", "dim", "vdim", "num_slots", "chunks")] + \
               [("eps", ctypes.c_float)]


def delta_chunkable(dtype, dim: int, vdim: int) -> bool:
    return dtype == torch.bfloat16 and dim % 8 == 0 and vdim % 8 == 0 and dim <= 128 and vdim <= 128


def delta_steps(dim: int, vdim: int) -> bool:
    """Whether a decode step of these sizes runs on the one-pass kernel, which also takes the gates' products and the convolution."""
    groups = vdim // 4
    return vdim % 4 == 0 and 0 < groups <= 256 and -(-dim // max(1, 256 // groups)) <= 16


def delta_rule(c, gate, ab, decay, dt, weight, state, at: StepRows, kv_heads: int, eps: float, y, conv=None, chunks=None):
    """Gated delta rule over rows q | k | v of ``c``: S <- g S, u = beta (v - S^T k), S <- S + k u^T, o = S^T q with unit q (times dim^-1/2) and
    k, g = exp(decay softplus(a + dt)), beta = sigmoid(b); y (R, heads * vdim) receives o / rms(o) * weight * silu(gate).  ``ab`` (R, 2 * heads)
    fp32: a | b; or, in a step of ``delta_steps`` sizes, the pair (input rows h, weights of a | b).  The states (slots, heads, dim, vdim) are
    read and left in their slots.  ``conv`` = (w (taps, channels), ring): single rows of ``delta_steps`` sizes pass the short convolution and
    silu here.  ``chunks`` = (offsets, number) of 64-token chunks (``StepBatch.chunk_ranges``): the tensor-core kernels for portions."""
    h = w_ab = None
    if isinstance(ab, tuple):
        h, w_ab = ab
        ab = None if c.is_cuda else h.float() @ w_ab.float().t()
    if not c.is_cuda:
        if conv is not None:
            c = mixer_torch.short_conv(c, conv[0], conv[1], at, True)
        return mixer_torch.delta_rule(c, gate, ab, decay, dt, weight, state, at, kv_heads, eps, y)
    slots, heads, dim, vdim = state.shape
    _req(state.dtype == torch.float32 and state.is_contiguous() and c.shape[1] == 2 * kv_heads * dim + heads * vdim and c.stride(1) == 1, "bad state")
    _req(at.state_slots.dtype == torch.int32 and at.positions.dtype == torch.int32 and decay.dtype == torch.float32 and dt.dtype == torch.float32
         and decay.numel() == heads and dt.numel() == heads, "bad inputs")
    _req(gate.shape == (c.shape[0], heads * vdim) and y.shape == gate.shape and gate.dtype == c.dtype and y.dtype == c.dtype
         and gate.stride(1) == 1 and y.stride(1) == 1 and weight.dtype == c.dtype and weight.numel() == vdim, "bad shapes")
    if ab is None:
        _req(h.dtype == c.dtype and w_ab.dtype == c.dtype and h.stride(1) == 1 and w_ab.shape == (2 * heads, h.shape[1])
             and at.cu is None and delta_steps(dim, vdim), "bad inputs of the gates")
    else:
        _req(ab.dtype == torch.float32 and ab.shape == (c.shape[0], 2 * heads) and ab.stride(1) == 1, "bad gates")
    w = ring = image = None
    if conv is not None:
        w, ring = conv
        _req(at.cu is None and delta_steps(dim, vdim) and w.is_contiguous() and w.dtype == c.dtype and ring.is_contiguous() and ring.dtype == c.dtype
             and ring.shape == (slots, *w.shape) and w.shape[1] == c.shape[1], "bad convolution")
    lib = _lib()
    if chunks is not None:
        _req(delta_chunkable(c.dtype, dim, vdim) and at.cu is not None, "sizes the chunked kernel does not take")
        _req(chunks[0].dtype == torch.int32 and chunks[0].numel() == at.state_slots.numel() + 1, "bad chunks")
        image = torch.empty(chunks[1] * heads * lib.b200_delta_image_bytes(), dtype=torch.uint8, device=c.device)
    ld = lambda t: 0 if t is None else t.stride(0)
    args = _DeltaArgs(_ptr(c), _ptr(gate), _ptr(ab), _ptr(h), _ptr(w_ab), _ptr(decay), _ptr(dt), _ptr(weight), _ptr(w), _ptr(ring), _ptr(y),
                      _ptr(state), _ptr(image), _ptr(at.state_slots), _ptr(at.cu), _ptr(at.positions), None if chunks is None else _ptr(chunks[0]),
                      _ptr(native.status_word(c.device)), ld(c), ld(gate), ld(ab), ld(h), ld(w_ab), ld(y), 0 if h is None else h.shape[1],
                      0 if w is None else w.shape[0], at.state_slots.numel(), c.shape[0], heads, kv_heads, dim, vdim, slots,
                      0 if chunks is None else chunks[1], float(eps))
    _check(lib.b200_delta(ctypes.byref(args), int(chunks is not None), _f32(c), _stream()), "delta_chunk" if chunks is not None else "delta")
    return y


DELTA_CHUNK = 64                 # tokens per chunk of the tensor-core kernels (csrc/delta.cu: DC)


# ------------------------------------------------------------------------- gated sublayers between group norms
class _GroupStart(ctypes.Structure):
    """csrc/group_norm.cu: GroupStart"""
    _fields_ = [(n, ctypes.c_void_p) for n in ("tokens", "embed", "bigram", "prev", "state_slots", "row_seq", "positions", "cu")] + \
               [(n, ctypes.c_longlong) for n in ("mul_prev", "mul_cur")] + \
               [(n, ctypes.c_int) for n in ("vocab", "buckets", "num_slots", "n_single", "portions")] + [("scale", ctypes.c_float)]


class _GroupSublayer(ctypes.Structure):
    """csrc/group_norm.cu: GroupSublayer"""
    _fields_ = [(n, ctypes.c_void_p) for n in ("y", "gate", "w_post", "ypos", "yweight")] + \
               [(n, ctypes.c_longlong) for n in ("ld_y", "ld_gate")] + [(n, ctypes.c_int) for n in ("ytop", "y_rows")]


class EmbeddingStart(NamedTuple):
    """x = embed[token] * scale, plus bigram[(previous token * mul_prev + token * mul_cur) mod buckets] (its last row for a sequence's first
    token); ``prev`` (slots, 1) int32 holds the sequences' last tokens."""
    embed: torch.Tensor
    scale: float
    bigram: torch.Tensor | None = None       # (buckets + 1, d)
    mul_prev: int = 0
    mul_cur: int = 0
    prev: torch.Tensor | None = None


class GatedOutput(NamedTuple):
    """What a gated sublayer adds to the residual stream: group_norm(y * sigmoid(gate)) * w_post."""
    y: torch.Tensor | ExpertOutputs
    gate: torch.Tensor                       # (R, d)
    w_post: torch.Tensor


def group_step(x, groups: int, eps: float, w=None, start: EmbeddingStart | None = None, batch=None, sub: GatedOutput | None = None, row_index=None):
    """One pass over the fp32 residual stream x (R, d): starts the rows of ``batch``, or adds a sublayer's output; returns
    h = group_norm(x) * w (no ``w``: None).  ``row_index``: h for these rows of x only, x itself stays as it is."""
    if not x.is_cuda:
        return mixer_torch.group_step(x, groups, eps, w, start, batch, sub, row_index)
    d = x.shape[1]
    rows = x.shape[0] if row_index is None else row_index.numel()
    act = w if w is not None else (start.embed if start is not None else sub.w_post)
    fits = lambda t: t is None or (t.dtype == act.dtype and t.is_contiguous() and t.shape[-1] == d)
    _req(x.dtype == torch.float32 and x.is_contiguous() and d % groups == 0 and fits(w), "bad residual stream")
    _req(row_index is None or (row_index.dtype == torch.int64 and row_index.is_contiguous() and start is None), "row_index must be int64")
    a = b = None
    if start is not None:
        _req(fits(start.embed) and fits(start.bigram) and batch.tokens.dtype == torch.int64 and batch.tokens.numel() == rows, "bad embedding")
        _req(start.bigram is None or (start.prev.dtype == torch.int32 and start.prev.is_contiguous()), "bad token state")
        a = _GroupStart(_ptr(batch.tokens), _ptr(start.embed), _ptr(start.bigram), _ptr(start.prev), _ptr(batch.state_slots), _ptr(batch.row_seq),
                        _ptr(batch.positions), _ptr(batch.cu), start.mul_prev, start.mul_cur, start.embed.shape[0],
                        0 if start.bigram is None else start.bigram.shape[0] - 1, 0 if start.prev is None else start.prev.shape[0], batch.n_single,
                        len(batch.portions), float(start.scale))
    if sub is not None:
        y, ex = (sub.y.y, sub.y) if isinstance(sub.y, ExpertOutputs) else (sub.y, None)
        _req(y.dtype == act.dtype and y.shape[1] == d and y.stride(1) == 1 and fits(sub.w_post) and sub.gate.dtype == act.dtype
             and sub.gate.shape == x.shape and sub.gate.stride(1) == 1, "bad sublayer output")
        _req(y.shape[0] == x.shape[0] if ex is None else (ex.z is None and ex.s is None and ex.pos.shape == ex.weight.shape and ex.pos.is_contiguous()
             and ex.weight.is_contiguous() and ex.scale == 1.0 and ex.pos.shape[0] == x.shape[0]), "bad expert outputs")
        b = _GroupSublayer(_ptr(y), _ptr(sub.gate), _ptr(sub.w_post), None if ex is None else _ptr(ex.pos), None if ex is None else _ptr(ex.weight),
                           y.stride(0), sub.gate.stride(0), 0 if ex is None else ex.pos.shape[1], y.shape[0])
    h = None if w is None else rows_buffer(rows, d, w.dtype, x.device)
    _check(_lib().b200_group_step(_ptr(x), _ref(a), _ref(b), _ptr(row_index), _ptr(w), _ptr(h), 0 if h is None else h.stride(0), float(eps), rows,
                                  x.shape[0], d, groups, _f32(act), _ptr(native.status_word(x.device)), _stream()), "group_step")
    return h
