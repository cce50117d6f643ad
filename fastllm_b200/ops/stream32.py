"""Operators of models whose residual stream is kept in fp32 (``csrc/stream32.cu``): token embedding plus sinusoidal or learned
positions with the first norm, RMSNorm of an fp32 row into the activation type, latent rows (norms, rotary key part) into their cache
slots, and the sub-layer's end: output norm, residual add and next norm, for a plain output or a mixture-of-experts combine, or for a
layer whose sub-layers stand side by side behind gates of their own.

CPU tensors evaluate the PyTorch definitions, which also serve the operator tests.
"""
from __future__ import annotations

import ctypes

import torch

from . import _lib
from .attention import ROPE_INTERLEAVED, ROPE_NEOX, apply_rope_ref
from .basic import _ptr, _stream

P, I, F, LL = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_longlong
_lib.register_sigs({
    "fb_rmsnorm32": [P, P, P, I, I, I, I, F, I, P],
    "fb_embed_pos_norm": [P, P, P, P, P, I, P, P, P, P, I, I, I, F, I, P],
    "fb_latent_post": [P, LL, I, I, I, I, I, I, I, I, I, I, I, I, P, P, P, P, I, P, P, P, P, P, I, LL, F, I, P],
    "fb_rope_heads": [P, P, LL, LL, I, I, I, I, I, I, I, P, P, P, I, I, P],
    "fb_gated_join": [P, P, P, I, P, LL, P, LL, P, P, P, P, LL, I, I, I, I, P, P, P, P, F, I, P],
    "fb_moe_combine_norm32": [P, P, P, F, P, P, P, P, P, I, I, I, F, F, P, P, I, P, I, P],
    "fb_moe_gather_scaled": [P, P, P, P, I, I, I, I, P],
    "fb_gather_rows": [P, P, P, I, I, P],
}, ["stream32"])


def act_code(dt: torch.dtype) -> int:
    return {torch.float16: 0, torch.bfloat16: 1, torch.float32: 2}[dt]


def _rms(x, w, eps):
    return x * torch.rsqrt(x.pow(2).mean(-1, keepdim=True) + eps) * w.float()


def sinusoid_inv_freq(width: int, base: float, device) -> torch.Tensor:
    """float64 [ceil(width / 2)]: base^(-2i / width)."""
    i = torch.arange(0, width, 2, dtype=torch.float64)
    return (base ** (-i / width)).to(device)


def embed_pos_norm(ids, positions, table, inv_freq, norm_w, eps: float, pos_table=None, add_vec=None):
    """fp32 residual ``table[ids] + positions`` and its RMSNorm in the table's type (``norm_w`` None: the residual itself in that type).
    Positions: ``inv_freq`` gives sines and cosines in alternating entries, ``pos_table`` learned rows; neither: none.  ``add_vec``: a row
    that every token gets."""
    T, H = ids.shape[0], table.shape[1]
    if not table.is_cuda:
        h = table[ids.long()].float()
        if inv_freq is not None:
            ang = positions.double()[:, None] * inv_freq[None, :]
            h = h + torch.stack([ang.sin(), ang.cos()], dim=-1).reshape(T, -1)[:, :H].float()
        if pos_table is not None:
            h = h + pos_table[positions.long()].float()
        if add_vec is not None:
            h = h + add_vec.float()
        return h, (_rms(h, norm_w, eps) if norm_w is not None else h).to(table.dtype)
    h = torch.empty((T, H), device=table.device, dtype=torch.float32)
    y = _out_rows(h, norm_w, table.dtype)
    rc = _lib.kernels().fb_embed_pos_norm(_ptr(ids), _ptr(positions), _ptr(table), _ptr(inv_freq), _ptr(pos_table), pos_table.shape[0] if pos_table is not None else 0,
                                          _ptr(add_vec), _ptr(norm_w), _ptr(h), _ptr(y if y is not h else None), T, H, table.shape[0], float(eps), act_code(table.dtype), _stream())
    _lib.check(rc, "fb_embed_pos_norm")
    return h, y


def _out_rows(h, norm_w, dtype):
    """Where the next reader's rows go: the fp32 residual itself when it reads it as it is in fp32."""
    return h if norm_w is None and dtype == torch.float32 else torch.empty(h.shape, device=h.device, dtype=dtype)


def rmsnorm32(x, w, eps: float):
    """RMSNorm of fp32 rows, returned in the type of ``w``."""
    if not x.is_cuda:
        return _rms(x, w, eps).to(w.dtype)
    M, H = x.shape
    y = torch.empty((M, H), device=x.device, dtype=w.dtype)
    rc = _lib.kernels().fb_rmsnorm32(_ptr(x), _ptr(w), _ptr(y), M, H, x.stride(0), H, float(eps), act_code(w.dtype), _stream())
    _lib.check(rc, "fb_rmsnorm32")
    return y


def layernorm(x, w, eps):
    """Layer norm without bias, fp32 rows."""
    d = x - x.mean(-1, keepdim=True)
    return d * torch.rsqrt(d.pow(2).mean(-1, keepdim=True) + eps) * w.float()


def latent_post(x, kv_col: int, kv_norm, rank: int, slots, pool, eps: float, lv: int | None = None, rot_col: int = 0, rot: int = 0, neox: bool = False, positions=None,
                cos=None, sin=None, q_norm=None, q_pad: int = 0, gate_col: int = 0, n_gates: int = 0):
    """What follows the merged projection ``x`` ``[T, ...]`` of latent attention, in one launch.  The cache rows ``slots`` of ``pool``
    ``[pages, page_len, 1, ld]`` (``slots`` < 0: the pool's spare last slot) become ``[RMSNorm(x[kv_col : + rank]) | 0]`` in the first ``lv``
    columns (default: all) and the rotated key part ``x[rot_col : + rot]`` behind them.  Returns (the normalised query latent, from column 0,
    ``[T, q_pad]`` or None without ``q_norm``; the head gates' logits ``x[gate_col : + n_gates]`` in fp32 or None)."""
    T, ld = x.shape[0], pool.shape[-1]
    lv = ld if lv is None else lv
    spare = pool.shape[0] * pool.shape[1] - 1
    q_rank = q_norm.shape[0] if q_norm is not None else 0
    cq = torch.empty((T, q_pad), device=x.device, dtype=x.dtype) if q_rank else None
    gates = torch.empty((T, n_gates), device=x.device, dtype=torch.float32) if n_gates else None
    if not pool.is_cuda:
        entry = torch.zeros((T, ld), dtype=pool.dtype)
        entry[:, :rank] = _rms(x[:, kv_col:kv_col + rank].float(), kv_norm, eps).to(pool.dtype)
        if rot:
            entry[:, lv:lv + rot] = apply_rope_ref(x[:, rot_col:rot_col + rot].unsqueeze(1), positions, cos, sin, ROPE_NEOX if neox else ROPE_INTERLEAVED, rot)[:, 0]
        pool.view(-1, ld).index_copy_(0, torch.where(slots >= 0, slots, torch.full_like(slots, spare)).long(), entry)
        if cq is not None:
            cq[:, q_rank:].zero_()
            cq[:, :q_rank] = _rms(x[:, :q_rank].float(), q_norm, eps).to(x.dtype)
        return cq, (gates.copy_(x[:, gate_col:gate_col + n_gates]) if gates is not None else None)
    rc = _lib.kernels().fb_latent_post(_ptr(x), x.stride(0), 0, q_rank, q_pad, kv_col, rank, lv, rot_col, rot, ld, int(neox), gate_col, n_gates, _ptr(q_norm), _ptr(kv_norm),
                                       _ptr(cos), _ptr(sin), cos.shape[0] if cos is not None else 0, _ptr(positions), _ptr(slots), _ptr(cq), _ptr(pool), _ptr(gates), T, spare,
                                       float(eps), act_code(pool.dtype), _stream())
    _lib.check(rc, "fb_latent_post")
    return cq, gates


def rope_heads(src, head_src: int, dst, head_dst: int, heads: int, rot: int, width: int, positions, cos, sin, neox: bool = False) -> None:
    """``dst[t, h * head_dst : + width] = src[t, h * head_src : + width]`` with the first ``rot`` dimensions of every head turned (CUDA tensors;
    ``src`` and ``dst`` start at the first head's dimensions; ``dst`` may be ``src``)."""
    rc = _lib.kernels().fb_rope_heads(_ptr(src), _ptr(dst), src.stride(0), dst.stride(0), src.shape[0], heads, head_src, head_dst, rot, width, int(neox), _ptr(positions),
                                      _ptr(cos), _ptr(sin), cos.shape[0], act_code(src.dtype), _stream())
    _lib.check(rc, "fb_rope_heads")


def gated_join(h, mixer, ff, w1, w2, eps: float, dtype, center: bool = True, embed=None):
    """The end of a layer whose mixer and feed-forward stand side by side: ``h += sigmoid(g1) * y1 + sigmoid(g2) * y2`` in place (fp32 rows), then
    ``(Norm(h) * w1, Norm(h) * w2)`` in the activation type (``w2`` None: None), a layer norm or (``center`` False) an RMS norm.
    ``mixer``: (y1, g1) or None; ``ff``: (rows, pos, weights, g2 in fp32) as the expert combine takes them (``pos`` None: the rows are y2
    itself) or None.  ``embed``: (table, ids) -- ``h`` starts as the tokens' embedding."""
    T, H = h.shape
    if not h.is_cuda:
        if embed is not None:
            h.copy_(embed[0][embed[1].long()])
        if mixer is not None:
            h += torch.sigmoid(mixer[1].float()) * mixer[0].float()
        if ff is not None:
            ys, pos, wts, g2 = ff
            y = ys.float()
            if pos is not None:
                p = pos.long()
                y = (y[p.clamp(min=0)] * torch.where(p >= 0, wts, torch.zeros_like(wts))[..., None]).sum(1)
            h += torch.sigmoid(g2.float()) * y
        norm = layernorm if center else _rms
        return norm(h, w1, eps).to(dtype), (norm(h, w2, eps).to(dtype) if w2 is not None else None)
    x1 = torch.empty((T, H), device=h.device, dtype=dtype)
    x2 = torch.empty_like(x1) if w2 is not None else None
    (table, ids), (y1, g1), (ys, pos, wts, g2) = embed or (None, None), mixer or (None, None), ff or (None,) * 4
    st = lambda t: t.stride(0) if t is not None else 0
    rc = _lib.kernels().fb_gated_join(_ptr(h), _ptr(table), _ptr(ids), table.shape[0] if table is not None else 0, _ptr(y1), st(y1), _ptr(g1), st(g1), _ptr(ys), _ptr(pos),
                                      _ptr(wts), _ptr(g2), st(g2), T, pos.shape[-1] if pos is not None else 1, H, int(center), _ptr(w1), _ptr(w2), _ptr(x1),
                                      _ptr(x2), float(eps), act_code(dtype), _stream())
    _lib.check(rc, "fb_gated_join")
    return x1, x2


def _start_args(start):
    """``start``: what opens a pass of looped layers, (embedding table or None, token ids, step vector)."""
    table, ids, vec = start if start is not None else (None, None, None)
    return _ptr(table), _ptr(ids if table is not None else None), table.shape[0] if table is not None else 0, _ptr(vec)


def moe_combine_norm(ys, pos, wts, wconst: float, shared, h, norm_w, alpha: float, eps: float, post_w=None, dtype=None, start=None):
    """``y = sum_k w_k * ys[pos[:, k]] + shared``, RMSNorm with ``post_w`` where the layer has an output norm, ``h += alpha * y`` in place
    (fp32), then RMSNorm(h) in the activation type ``dtype`` (``norm_w`` None: h itself in it).  ``wts`` None: every weight is
    ``wconst``.  ``pos`` < 0: the pair is not held here.  ``start``: see ``add_norm``."""
    T, H = h.shape
    topk = pos.shape[-1]
    dtype = dtype or (norm_w.dtype if norm_w is not None else ys.dtype)
    if not h.is_cuda:
        w = wts if wts is not None else torch.full((T, topk), wconst)
        p = pos.reshape(T, topk).long()
        y = (ys.float()[p.clamp(min=0)] * torch.where(p >= 0, w, torch.zeros_like(w))[..., None]).sum(1)
        if shared is not None:
            y = y + shared.float()
        return add_norm(h, y, post_w, norm_w, eps, alpha, dtype, start)
    out = _out_rows(h, norm_w, dtype)
    rc = _lib.kernels().fb_moe_combine_norm32(_ptr(ys), _ptr(pos), _ptr(wts), float(wconst), _ptr(shared), _ptr(h), _ptr(post_w), _ptr(norm_w),
                                              _ptr(out if out is not h else None), T, topk, H, float(alpha), float(eps), *_start_args(start), act_code(dtype), _stream())
    _lib.check(rc, "fb_moe_combine_norm32")
    return out


def add_norm(h, y, post_w, norm_w, eps: float, alpha: float = 1.0, dtype=None, start=None):
    """``h += alpha * RMSNorm(y)`` in place (fp32 rows; ``post_w`` None: y itself; ``y`` None: nothing), then RMSNorm(h) in the activation
    type (``norm_w`` None: h itself in that type).  ``start``: (embedding table or None, token ids, vector) -- the residual also gets
    the vector and the token's embedding before that norm, which is how a pass of looped layers opens."""
    dtype = dtype or (y.dtype if y is not None else norm_w.dtype)
    if not h.is_cuda:
        if y is not None:
            h += alpha * (_rms(y.float(), post_w, eps) if post_w is not None else y.float())
        if start is not None:
            table, ids, vec = start
            h += (table[ids.long()].float() if table is not None else 0.0) + vec.float()
        return (_rms(h, norm_w, eps) if norm_w is not None else h).to(dtype)
    out = _out_rows(h, norm_w, dtype)
    rc = _lib.kernels().fb_moe_combine_norm32(_ptr(y), _ptr(None), _ptr(None), 1.0, _ptr(None), _ptr(h), _ptr(post_w), _ptr(norm_w),
                                              _ptr(out if out is not h else None), h.shape[0], 1, h.shape[1], float(alpha), float(eps), *_start_args(start), act_code(dtype),
                                              _stream())
    _lib.check(rc, "fb_moe_combine_norm32")
    return out


def moe_gather_scaled(x32, pos, wts, xs) -> None:
    """``xs[pos[t, k]] = wts[t, k] * x32[t]`` for the pairs held here: fp32 rows to the activation type, rounded once."""
    T, topk = pos.shape
    rc = _lib.kernels().fb_moe_gather_scaled(_ptr(x32), _ptr(pos), _ptr(wts), _ptr(xs), T, topk, x32.shape[1], act_code(xs.dtype), _stream())
    _lib.check(rc, "fb_moe_gather_scaled")


def gather_rows(src, idx):
    """``src[idx]`` for rows of a multiple of 16 bytes."""
    if not src.is_cuda:
        return src.index_select(0, idx)
    out = torch.empty((idx.shape[0], src.shape[1]), device=src.device, dtype=src.dtype)
    rc = _lib.kernels().fb_gather_rows(_ptr(src), _ptr(idx), _ptr(out), idx.shape[0], src.shape[1] * src.element_size(), _stream())
    _lib.check(rc, "fb_gather_rows")
    return out
