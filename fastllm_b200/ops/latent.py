"""Latent attention without positions: every head's keys and values are linear in one cached latent row per token.

Two evaluations of the same mixer, chosen per request of a batch:

* *absorbed* (decoded tokens, short portions): queries are multiplied into the latent space, every row attends to the cached
  latents themselves (``csrc/attn_mla.cu``), the result is multiplied by the value projection with the output gate in its epilogue;
* *expanded* (prompt chunks): the latents the chunk's queries see are gathered once, one GEMM expands them to keys and values, and
  the windowed prefill kernel (``csrc/attn_window.cu``) runs on plain heads, output gate in its epilogue.

Other element types or widths (float32; latents beyond the decode kernel) run every row through ``csrc/full32.cu``.  CPU tensors
evaluate the PyTorch definition.
"""
from __future__ import annotations

import ctypes

import numpy as np
import torch

from . import _lib
from . import basic as B
from . import stream32 as S
from .attention import mla_decode
from .basic import _ptr, _stream, dtype_code

P, I, F, LL = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_longlong
_lib.register_sigs({
    "fb_latent_attn32": [P, P, P, P, P, I, I, I, I, I, I, I, F, I, P],
    "fb_attn_window": [P, LL, I, P, LL, P, LL, I, P, LL, P, LL, P, I, I, I, I, I, F, I, P],
}, ["full32", "attn_window"])

ABSORB_ROWS = 16                 # requests that bring at most this many tokens attend in the latent space
EXPAND_BYTES = 2 << 30           # scratch keys and values of one expanded group of requests
_MAX_MLA_ROWS = 1024             # requests per call of the latent decode kernel


def _round8(n: int) -> int:
    return (n + 7) // 8 * 8


class LatentWeights:
    """One latent-attention layer.  ``dim`` / ``vdim`` / ``ld`` are the stored widths (multiples of 8, padded with zero rows and
    columns), ``rank`` the latent's own width."""

    def __init__(self):
        self.heads = self.dim = self.vdim = self.rank = self.ld = 0
        self.window = 0
        self.scale = 1.0
        self.in_proj = None      # rows [queries | output gate | latent]
        self.kv_norm = None
        self.w_ukv = None        # [heads * (dim + vdim), ld]: keys of all heads, then values (the expanding GEMM)
        self.w_uk_t = None       # [heads, ld, dim]   queries -> latent space
        self.w_uv = None         # [heads, vdim, ld]  latent space -> values
        self.has_gate = True

    @property
    def gate_col(self) -> int:
        return self.heads * self.dim

    @property
    def latent_col(self) -> int:
        return self.heads * (self.dim + (self.vdim if self.has_gate else 0))


def _pad_heads(w, heads: int, width: int):
    """[heads * n, K] -> [heads * width, K] with zero rows behind every head's own."""
    n = w.shape[0] // heads
    if n == width:
        return w
    out = torch.zeros((heads, width, w.shape[1]), dtype=w.dtype, device=w.device)
    out[:, :n] = w.reshape(heads, n, w.shape[1])
    return out.reshape(heads * width, w.shape[1])


def pad_rows(w, mult: int):
    extra = -w.shape[0] % mult
    return w if extra == 0 else torch.cat([w, torch.zeros((extra, *w.shape[1:]), dtype=w.dtype, device=w.device)], dim=0)


def pad_cols(w, mult: int):
    extra = -w.shape[1] % mult
    return w if extra == 0 else torch.cat([w, torch.zeros((w.shape[0], extra), dtype=w.dtype, device=w.device)], dim=1)


def build(spec, q, g, dkv, kv_norm, uk, uv):
    """(LatentWeights without ``in_proj``, merged input projection matrix) from the layer's matrices."""
    w = LatentWeights()
    H = w.heads = spec.heads
    w.dim, w.vdim, w.rank, w.ld = _round8(spec.dim), _round8(spec.vdim), spec.kv_rank, _round8(spec.kv_rank)
    w.window, w.scale = int(spec.window or 0), float(spec.scale)
    w.has_gate = g is not None
    parts = [_pad_heads(q, H, w.dim)] + ([_pad_heads(g, H, w.vdim)] if w.has_gate else []) + [pad_rows(dkv, 8)]
    w.kv_norm = kv_norm
    uk, uv = pad_cols(_pad_heads(uk, H, w.dim), 8), pad_cols(_pad_heads(uv, H, w.vdim), 8)
    w.w_ukv = pad_rows(torch.cat([uk, uv], dim=0), 32).contiguous()
    w.w_uk_t = uk.reshape(H, w.dim, w.ld).transpose(1, 2).contiguous()
    w.w_uv = uv.reshape(H, w.vdim, w.ld).contiguous()
    return w, pad_rows(torch.cat(parts, dim=0), 32)


def pad_out_proj(o, spec):
    """Output projection [width, heads * vdim] with zero columns where the heads are padded."""
    return _pad_heads(o.t().contiguous(), spec.heads, _round8(spec.vdim)).t().contiguous()


# ---------------------------------------------------------------------------------------------------
# batch plans: which rows are absorbed, which requests are expanded; shared by all layers with the same window
# ---------------------------------------------------------------------------------------------------
class _Group:
    """Requests whose keys are expanded together."""

    def __init__(self, key_idx, blocks, n_blocks):
        self.key_idx, self.blocks, self.n_blocks = key_idx, blocks, n_blocks


class LatentPlan:
    def __init__(self):
        self.rows = None             # int64 rows of the packed batch that are absorbed (None: all of them)
        self.n_rows = 0
        self.page_table = None       # [n_rows, P] and [n_rows]: every absorbed row is a request of its own
        self.kv_lens = None
        self.groups: list[_Group] = []


def _row_plan(fb, reqs, cu, dev):
    """Page-table rows and visible lengths of all rows of the requests ``reqs``."""
    owner = np.concatenate([np.full(cu[b + 1] - cu[b], b, dtype=np.int64) for b in reqs])
    rows = np.concatenate([np.arange(cu[b], cu[b + 1], dtype=np.int64) for b in reqs])
    return torch.from_numpy(owner).to(dev, non_blocking=True), torch.from_numpy(rows).to(dev, non_blocking=True)


def build_plan(fb, window: int, page_len: int, expand: bool, key_bytes: int) -> LatentPlan:
    pl = LatentPlan()
    if fb.is_decode:
        pl.page_table, pl.kv_lens, pl.n_rows = fb.page_table, fb.kv_lens, fb.page_table.shape[0]
        return pl
    dev = fb.page_table.device
    cu = fb.cu_q_host if fb.cu_q_host is not None else fb.cu_q.tolist()
    lens = fb.kv_lens_host if fb.kv_lens_host is not None else fb.kv_lens.tolist()
    reqs = [b for b in range(len(cu) - 1) if cu[b + 1] > cu[b]]
    long = [b for b in reqs if expand and cu[b + 1] - cu[b] > ABSORB_ROWS]
    short = [b for b in reqs if b not in set(long)]
    if short:
        owner, rows = _row_plan(fb, short, cu, dev)
        pl.n_rows = rows.shape[0]
        pl.page_table = fb.page_table.index_select(0, owner)
        seen = fb.positions + 1
        pl.kv_lens = seen.to(torch.int32) if not long else seen.index_select(0, rows).to(torch.int32)
        pl.rows = rows if long else None
    group, base = [], 0
    pending: list = []

    def flush():
        if not pending:
            return
        owner = np.concatenate([np.full(n, b, dtype=np.int64) for b, _, n in pending])
        pos = np.concatenate([np.arange(k, k + n, dtype=np.int64) for _, k, n in pending])
        meta = torch.from_numpy(np.stack([owner, pos])).to(dev, non_blocking=True)
        pages = fb.page_table[meta[0], torch.div(meta[1], page_len, rounding_mode="floor")].long()
        blocks = sorted(group, key=lambda t: -(min(t[1] + t[2] - t[4], (window or 1 << 30) + t[2])))      # most keys first
        pl.groups.append(_Group(pages * page_len + meta[1] % page_len, torch.tensor(blocks, dtype=torch.int32).to(dev, non_blocking=True), len(blocks)))

    for b in long:
        n, start = cu[b + 1] - cu[b], lens[b] - (cu[b + 1] - cu[b])
        k0 = max(0, start - window + 1) if window else 0
        if pending and (base + lens[b] - k0) * key_bytes > EXPAND_BYTES:
            flush()
            group, pending, base = [], [], 0
        for q0 in range(0, n, 256):
            group.append((cu[b] + q0, start + q0, min(256, n - q0), base, k0, 0))
        pending.append((b, k0, lens[b] - k0))
        base += lens[b] - k0
    flush()
    return pl


def _plan(fb, lw, page_len: int, expand: bool) -> LatentPlan:
    key_bytes = lw.heads * (lw.dim + lw.vdim) * 2
    key = (lw.window, expand, key_bytes)
    cache = fb.__dict__.setdefault("_latent_plans", {})
    if key not in cache:
        cache[key] = build_plan(fb, lw.window, page_len, expand, key_bytes)
    return cache[key]


# ---------------------------------------------------------------------------------------------------
def decode_kernel_ok(lw, dtype, page_len: int) -> bool:
    return dtype in (torch.float16, torch.bfloat16) and lw.ld <= 512 and page_len == 128


def expand_ok(lw, dtype) -> bool:
    if dtype not in (torch.float16, torch.bfloat16):
        return False
    ok = lw.__dict__.get("_expand_ok")
    if ok is None:
        ok = lw._expand_ok = bool(_lib.kernels()._lib.fb_attn_window_supported(lw.dim, lw.vdim))
    return ok


def _absorbed(lw, q, gate, pool, page_table, kv_lens, out):
    """Rows ``q`` [n, heads * dim] (row stride free) against their own page-table rows; the gated values go to ``out`` [n, heads * vdim]."""
    n, H = q.shape[0], lw.heads
    q_lat = torch.empty((n, H, lw.ld), device=q.device, dtype=q.dtype)
    B.linear_batched(q, lw.w_uk_t, H, lw.dim, q_lat.view(n, H * lw.ld), lw.ld)
    if decode_kernel_ok(lw, q.dtype, pool.shape[1]):
        o_lat = torch.cat([mla_decode(q_lat[i:i + _MAX_MLA_ROWS], pool, page_table[i:i + _MAX_MLA_ROWS], kv_lens[i:i + _MAX_MLA_ROWS], lw.scale,
                                      window=lw.window) for i in range(0, n, _MAX_MLA_ROWS)]) if n > _MAX_MLA_ROWS else \
            mla_decode(q_lat, pool, page_table, kv_lens, lw.scale, window=lw.window)
    else:
        o_lat = torch.empty_like(q_lat)
        rc = _lib.kernels().fb_latent_attn32(_ptr(q_lat), _ptr(pool), _ptr(o_lat), _ptr(page_table), _ptr(kv_lens), n, H, lw.rank, lw.ld,
                                             page_table.stride(0), pool.shape[1], lw.window, lw.scale, S.act_code(q.dtype), _stream())
        _lib.check(rc, "fb_latent_attn32")
    B.linear_batched(o_lat.view(n, H * lw.ld), lw.w_uv, H, lw.ld, out, lw.vdim, gate=gate)


def window_attention(lw, grp, q, gate, kv, out):
    """Prefill kernel over one group's expanded keys and values ``kv`` [n_keys, >= heads * (dim + vdim)]."""
    H = lw.heads
    k, v = kv[:, :H * lw.dim], kv[:, H * lw.dim:]
    rc = _lib.kernels().fb_attn_window(_ptr(q), q.stride(0), q.shape[0], _ptr(k), kv.stride(0), _ptr(v), kv.stride(0), kv.shape[0], _ptr(out),
                                       out.stride(0), _ptr(gate), gate.stride(0) if gate is not None else 0, _ptr(grp.blocks), grp.n_blocks,
                                       H, lw.dim, lw.vdim, lw.window, lw.scale, dtype_code(q.dtype), _stream())
    _lib.check(rc, "fb_attn_window")


def attention(lw, proj, pool, fb):
    """``proj`` ``[T, >= latent_col]`` (queries and gate columns; the latents are in ``pool`` already) -> gated heads ``[T, heads * vdim]``."""
    T, H = proj.shape[0], lw.heads
    q = proj[:, :H * lw.dim]
    gate = proj[:, lw.gate_col:lw.gate_col + H * lw.vdim] if lw.has_gate else None
    if not proj.is_cuda:
        return attention_ref(lw, q, gate, pool, fb)
    out = torch.empty((T, H * lw.vdim), device=proj.device, dtype=proj.dtype)
    pl = _plan(fb, lw, pool.shape[1], expand_ok(lw, proj.dtype) and not fb.is_decode)
    if pl.n_rows and pl.rows is None:
        _absorbed(lw, q, gate, pool, pl.page_table, pl.kv_lens, out)
    elif pl.n_rows:
        part = torch.empty((pl.n_rows, H * lw.vdim), device=proj.device, dtype=proj.dtype)
        sub = proj.index_select(0, pl.rows)
        _absorbed(lw, sub[:, :H * lw.dim], sub[:, lw.gate_col:lw.gate_col + H * lw.vdim] if lw.has_gate else None, pool, pl.page_table,
                  pl.kv_lens, part)
        out.index_copy_(0, pl.rows, part)
    for grp in pl.groups:
        window_attention(lw, grp, q, gate, B.linear(S.gather_rows(pool.view(-1, lw.ld), grp.key_idx), lw.w_ukv), out)
    return out


def attention_ref(lw, q, gate, pool, fb):
    """PyTorch evaluation over the paged latents (CPU tensors)."""
    T, H, D, V = q.shape[0], lw.heads, lw.dim, lw.vdim
    page_len = pool.shape[1]
    cu = fb.cu_q_host if fb.cu_q_host is not None else fb.cu_q.tolist()
    out = torch.zeros((T, H, V), dtype=torch.float32)
    wk = lw.w_ukv[:H * D].float().reshape(H, D, lw.ld)
    wv = lw.w_ukv[H * D:H * (D + V)].float().reshape(H, V, lw.ld)
    for b, L in enumerate(fb.kv_lens.tolist()):
        r0, r1 = cu[b], cu[b + 1]
        if r1 == r0 or L == 0:
            continue
        npg = (L + page_len - 1) // page_len
        c = pool[fb.page_table[b, :npg].long()].reshape(-1, lw.ld)[:L].float()
        qpos = torch.arange(L - (r1 - r0), L)[:, None]
        kpos = torch.arange(L)[None, :]
        see = kpos <= qpos
        if lw.window:
            see = see & (kpos > qpos - lw.window)
        qh = q[r0:r1].float().reshape(-1, H, D)
        s = torch.einsum("qhd,khd->hqk", qh, torch.einsum("kr,hdr->khd", c, wk)) * lw.scale
        p = torch.softmax(s.masked_fill(~see, float("-inf")), dim=-1)
        out[r0:r1] = torch.einsum("hqk,khv->qhv", p, torch.einsum("kr,hvr->khv", c, wv))
    o = out.reshape(T, H * V)
    if gate is not None:
        o = o * torch.sigmoid(gate.float())
    return o.to(q.dtype)
