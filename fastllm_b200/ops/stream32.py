"""Operators of models whose residual stream is kept in fp32 (``csrc/stream32.cu``): token embedding plus sinusoidal or learned
positions with the first norm, RMSNorm of an fp32 row into the activation type, RMSNorm of a latent row into its cache slot, and the
sub-layer's end: output norm, residual add and next norm, for a plain output or a mixture-of-experts combine.

CPU tensors evaluate the PyTorch definitions, which also serve the operator tests.
"""
from __future__ import annotations

import ctypes

import torch

from . import _lib
from .basic import _ptr, _stream

P, I, F, LL = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_longlong
_lib.register_sigs({
    "fb_rmsnorm32": [P, P, P, I, I, I, I, F, I, P],
    "fb_embed_pos_norm": [P, P, P, P, P, I, P, P, P, P, I, I, I, F, I, P],
    "fb_latent_norm": [P, I, P, P, P, I, I, I, LL, F, I, P],
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


def latent_norm(x, w, slots, pool, rank: int, eps: float) -> None:
    """RMSNorm over the first ``rank`` columns of ``x`` ``[T, >= rank]`` into the cache rows ``slots`` of ``pool``
    ``[pages, page_len, 1, ld]`` (entry columns beyond ``rank`` are zero; rows with ``slots`` < 0 go to the pool's spare last slot)."""
    ld = pool.shape[-1]
    flat = pool.view(-1, ld)
    spare = flat.shape[0] - 1
    if not pool.is_cuda:
        y = _rms(x[:, :rank].float(), w[:rank], eps).to(pool.dtype)
        entry = torch.zeros((x.shape[0], ld), dtype=pool.dtype)
        entry[:, :rank] = y
        flat.index_copy_(0, torch.where(slots >= 0, slots, torch.full_like(slots, spare)).long(), entry)
        return
    rc = _lib.kernels().fb_latent_norm(_ptr(x), x.stride(0), _ptr(w), _ptr(slots), _ptr(pool), x.shape[0], rank, ld, spare, float(eps),
                                       act_code(pool.dtype), _stream())
    _lib.check(rc, "fb_latent_norm")


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
