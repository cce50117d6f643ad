"""Latent attention: every head's keys and values are linear in one cached latent row per token.  Where the layer has positions, a rotated
key part that all heads share is cached behind the latent (``[latent | 0 | rotated part]``); the queries may come through a latent of
their own, and the output gate is one per element or one per head.

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
from .attention import ROPE_INTERLEAVED, ROPE_NEOX, apply_rope_ref, mla_decode
from .basic import _ptr, _stream, dtype_code

P, I, F, LL = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_longlong
_lib.register_sigs({
    "fb_latent_attn32": [P, P, P, P, P, I, I, I, I, I, I, I, I, F, P, I, P],
    "fb_attn_window": [P, LL, I, I, P, LL, P, LL, P, LL, I, P, LL, P, LL, P, LL, P, I, I, I, I, I, I, F, I, P],
    "fb_attn_window_supported": [I, I, I],
}, ["full32", "attn_window"])

ABSORB_ROWS = 16                 # requests that bring at most this many tokens attend in the latent space
EXPAND_BYTES = 2 << 30           # scratch keys and values of one expanded group of requests
_MAX_MLA_ROWS = 1024             # requests per call of the latent decode kernel


def _round8(n: int) -> int:
    return (n + 7) // 8 * 8


def stored_widths(spec) -> tuple[int, int]:
    """Columns of a cached row: the latent's (values end at a tile where something follows them) and the rotated key part's."""
    return ((spec.kv_rank + 63) // 64 * 64, _round8(spec.rot_dim)) if spec.rot_dim else (_round8(spec.kv_rank), 0)


class LatentWeights:
    """One latent-attention layer.  ``dim`` / ``vdim`` are the stored widths (multiples of 8, padded with zero rows and columns) of a head's
    own query / key dimensions and values, ``rank`` the latent's own width.  A cached row is ``ld`` wide: ``lv`` columns of latent (padded), then
    ``rd`` of the rotated part (``rot`` of them used)."""

    def __init__(self):
        self.heads = self.dim = self.vdim = self.rank = self.lv = self.ld = 0
        self.rot = self.rd = 0
        self.neox = False
        self.window = 0
        self.scale = 1.0
        self.in_proj = None      # rows [queries or their latent | output gate | latent | rotated key part | the layer's further rows]
        self.q_up = None         # queries from their normalised latent, where they have one (``q_pad`` columns)
        self.q_norm = None
        self.q_pad = 0
        self.kv_norm = None
        self.w_ukv = None        # [heads * (dim + vdim), lv]: keys of all heads, then values (the expanding GEMM)
        self.w_uk_t = None       # [heads, lv, dim]   queries -> latent space
        self.w_uv = None         # [heads, vdim, lv]  latent space -> values
        self.gate = "elem"       # "elem": one per element, "head": one per head, "": none
        self.more_col = 0        # first of the further rows

    @property
    def hd(self) -> int:
        """Columns from one query head to the next: its own dimensions, then the rotated ones."""
        return self.dim + self.rd

    @property
    def gate_col(self) -> int:
        return self.q_pad if self.q_norm is not None else self.heads * self.hd

    @property
    def n_gates(self) -> int:
        return self.heads if self.gate == "head" else 0

    @property
    def latent_col(self) -> int:
        return self.gate_col + (self.heads * self.vdim if self.gate == "elem" else _round8(self.n_gates))

    @property
    def rot_col(self) -> int:
        return self.latent_col + _round8(self.rank)


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


def _head_rows(q, heads: int, parts):
    """Rows of heads laid out as ``parts`` [(width, stored width), ...], every part padded with zero rows."""
    q = q.reshape(heads, -1, q.shape[1])
    out = [_pad_part(x, p) for x, p in zip(q.split([n for n, _ in parts], dim=1), [p for _, p in parts])]
    return torch.cat(out, dim=1).reshape(-1, q.shape[2])


def _pad_part(x, rows: int):
    """[heads, n, K] -> [heads, rows, K]"""
    return torch.nn.functional.pad(x, (0, 0, 0, rows - x.shape[1]))


def build(spec, q, g, dkv, kv_norm, uk, uv, uq=None, q_norm=None, more=()):
    """(LatentWeights without ``in_proj`` and ``q_up``, merged input projection matrix, matrix of ``q_up`` or None) from the layer's matrices.
    ``uq`` / ``q_norm``: ``q`` projects to the queries' latent.  ``more``: matrices that read the same input."""
    w = LatentWeights()
    H = w.heads = spec.heads
    w.dim, w.vdim, w.rank = _round8(spec.dim), _round8(spec.vdim), spec.kv_rank
    w.rot, (w.lv, w.rd) = spec.rot_dim, stored_widths(spec)
    w.neox = bool(spec.rope and spec.rope.get("mode") == "neox")
    w.ld = w.lv + w.rd
    w.window, w.scale = int(spec.window or 0), float(spec.scale)
    w.gate = spec.gate if g is not None else ""
    heads = lambda m: _head_rows(m, H, [(spec.dim, w.dim), (spec.rot_dim, w.rd)])
    if uq is not None:
        w.q_norm, w.q_pad = q_norm, _round8(q.shape[0])
        parts = [pad_rows(q, 8)]
    else:
        parts = [heads(q)]
    if g is not None:
        parts.append(_pad_heads(g, H, w.vdim) if w.gate == "elem" else pad_rows(g, 8))
    parts += [pad_rows(dkv[:w.rank], 8)] + ([pad_rows(dkv[w.rank:], 8)] if w.rot else [])
    w.more_col = sum(m.shape[0] for m in parts)
    w.kv_norm = kv_norm
    uk, uv = (torch.nn.functional.pad(_pad_heads(m, H, n), (0, w.lv - w.rank)) for m, n in ((uk, w.dim), (uv, w.vdim)))
    w.w_ukv = pad_rows(torch.cat([uk, uv], dim=0), 32).contiguous()
    w.w_uk_t = uk.reshape(H, w.dim, w.lv).transpose(1, 2).contiguous()
    w.w_uv = uv.reshape(H, w.vdim, w.lv).contiguous()
    return w, pad_rows(torch.cat([*parts, *more], dim=0), 32), pad_cols(pad_rows(heads(uq), 32), 8).contiguous() if uq is not None else None


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
    return dtype in (torch.float16, torch.bfloat16) and lw.lv <= 512 and lw.ld <= 576 and page_len == 128


def expand_ok(lw, dtype) -> bool:
    if dtype not in (torch.float16, torch.bfloat16):
        return False
    ok = lw.__dict__.get("_expand_ok")
    if ok is None:
        ok = lw._expand_ok = bool(_lib.kernels()._lib.fb_attn_window_supported(lw.dim, lw.rd, lw.vdim))
    return ok


def post(lw, proj, fb, pool, rope, eps: float):
    """Latent row (and rotated key part) of every token into its cache slot; returns (queries [T, heads * hd] -- not rotated yet --, fp32 logits
    of the head gates or None).  ``rope``: (cos, sin) tables or None."""
    cos, sin = rope or (None, None)
    cq, gates = S.latent_post(proj, lw.latent_col, lw.kv_norm, lw.rank, fb.slots, pool, eps, lw.lv, lw.rot_col, lw.rot, lw.neox, fb.positions, cos, sin, lw.q_norm, lw.q_pad,
                              lw.gate_col, lw.n_gates)
    return (lw.q_up(cq) if cq is not None else proj)[:, :lw.heads * lw.hd], gates


def _absorbed(lw, q, gate, head_gate, pool, page_table, kv_lens, out, positions, rope):
    """Rows ``q`` [n, heads * hd] (row stride free) against their own page-table rows; the gated values go to ``out`` [n, heads * vdim]."""
    n, H = q.shape[0], lw.heads
    q_lat = torch.empty((n, H, lw.ld), device=q.device, dtype=q.dtype)
    B.linear_batched(q, lw.w_uk_t, H, lw.hd, q_lat.view(n, H * lw.ld), lw.ld)
    if lw.rd:
        S.rope_heads(q[:, lw.dim:], lw.hd, q_lat.view(n, H * lw.ld)[:, lw.lv:], lw.ld, H, lw.rot, lw.rd, positions, *rope, lw.neox)
    if decode_kernel_ok(lw, q.dtype, pool.shape[1]):
        part = lambda i, j: mla_decode(q_lat[i:j], pool, page_table[i:j], kv_lens[i:j], lw.scale, lora=lw.lv, window=lw.window,
                                       head_gate=head_gate[i:j] if head_gate is not None else None)
        o_lat = part(0, n) if n <= _MAX_MLA_ROWS else torch.cat([part(i, i + _MAX_MLA_ROWS) for i in range(0, n, _MAX_MLA_ROWS)])
    else:
        o_lat = torch.empty((n, H, lw.lv), device=q.device, dtype=q.dtype)
        rc = _lib.kernels().fb_latent_attn32(_ptr(q_lat), _ptr(pool), _ptr(o_lat), _ptr(page_table), _ptr(kv_lens), n, H, lw.ld, lw.lv, lw.ld,
                                             page_table.stride(0), pool.shape[1], lw.window, lw.scale, _ptr(head_gate), S.act_code(q.dtype), _stream())
        _lib.check(rc, "fb_latent_attn32")
    B.linear_batched(o_lat.view(n, H * lw.lv), lw.w_uv, H, lw.lv, out, lw.vdim, gate=gate)


def window_attention(lw, grp, q, gate, kv, out, head_gate=None, shared=None):
    """Prefill kernel over one group's expanded keys and values ``kv`` [n_keys, >= heads * (dim + vdim)]; ``shared``: [n_keys, rd] rotated key
    parts."""
    H = lw.heads
    k, v = kv[:, :H * lw.dim], kv[:, H * lw.dim:]
    st = lambda t: t.stride(0) if t is not None else 0
    rc = _lib.kernels().fb_attn_window(_ptr(q), q.stride(0), lw.hd, q.shape[0], _ptr(k), kv.stride(0), _ptr(v), kv.stride(0), _ptr(shared), st(shared), kv.shape[0],
                                       _ptr(out), out.stride(0), _ptr(gate), st(gate), _ptr(head_gate), st(head_gate), _ptr(grp.blocks), grp.n_blocks,
                                       H, lw.dim, lw.rd, lw.vdim, lw.window, lw.scale, dtype_code(q.dtype), _stream())
    _lib.check(rc, "fb_attn_window")


def attention(lw, proj, pool, fb, q=None, head_gate=None, rope=None):
    """``proj`` (elementwise gate columns; the new latent rows are in ``pool`` already), ``q`` and ``head_gate`` as ``post`` returned them (``q``
    None: the first columns of ``proj``) -> gated heads ``[T, heads * vdim]``.  May rotate the queries in place."""
    T, H = proj.shape[0], lw.heads
    q = proj[:, :H * lw.hd] if q is None else q
    gate = proj[:, lw.gate_col:lw.gate_col + H * lw.vdim] if lw.gate == "elem" else None
    if not proj.is_cuda:
        return attention_ref(lw, q, gate, pool, fb, head_gate, rope)
    out = torch.empty((T, H * lw.vdim), device=proj.device, dtype=proj.dtype)
    pl = _plan(fb, lw, pool.shape[1], expand_ok(lw, proj.dtype) and not fb.is_decode)
    if pl.n_rows and pl.rows is None:
        _absorbed(lw, q, gate, head_gate, pool, pl.page_table, pl.kv_lens, out, fb.positions, rope)
    elif pl.n_rows:
        part = torch.empty((pl.n_rows, H * lw.vdim), device=proj.device, dtype=proj.dtype)
        pick = lambda t: t.index_select(0, pl.rows) if t is not None else None
        _absorbed(lw, pick(q), pick(gate), pick(head_gate), pool, pl.page_table, pl.kv_lens, part, pick(fb.positions), rope)
        out.index_copy_(0, pl.rows, part)
    if pl.groups and lw.rd:
        qr = q[:, lw.dim:]
        S.rope_heads(qr, lw.hd, qr, lw.hd, H, lw.rot, lw.rd, fb.positions, *rope, lw.neox)
    for grp in pl.groups:
        rows = S.gather_rows(pool.view(-1, lw.ld), grp.key_idx)
        window_attention(lw, grp, q, gate, B.linear(rows[:, :lw.lv], lw.w_ukv), out, head_gate, rows[:, lw.lv:] if lw.rd else None)
    return out


def attention_ref(lw, q, gate, pool, fb, head_gate=None, rope=None):
    """PyTorch evaluation over the paged latents (CPU tensors)."""
    T, H, D, V = q.shape[0], lw.heads, lw.dim, lw.vdim
    page_len = pool.shape[1]
    cu = fb.cu_q_host if fb.cu_q_host is not None else fb.cu_q.tolist()
    out = torch.zeros((T, H, V), dtype=torch.float32)
    wk = lw.w_ukv[:H * D].float().reshape(H, D, lw.lv)
    wv = lw.w_ukv[H * D:H * (D + V)].float().reshape(H, V, lw.lv)
    q = q.reshape(T, H, lw.hd).float()
    if lw.rot:
        q = torch.cat([q[..., :D], apply_rope_ref(q[..., D:], fb.positions, *rope, ROPE_NEOX if lw.neox else ROPE_INTERLEAVED, lw.rot)], dim=-1)
    for b, L in enumerate(fb.kv_lens.tolist()):
        r0, r1 = cu[b], cu[b + 1]
        if r1 == r0 or L == 0:
            continue
        npg = (L + page_len - 1) // page_len
        rows = pool[fb.page_table[b, :npg].long()].reshape(-1, lw.ld)[:L].float()
        c, kr = rows[:, :lw.lv], rows[:, lw.lv:]
        qpos = torch.arange(L - (r1 - r0), L)[:, None]
        kpos = torch.arange(L)[None, :]
        see = kpos <= qpos
        if lw.window:
            see = see & (kpos > qpos - lw.window)
        s = torch.einsum("qhd,khd->hqk", q[r0:r1, :, :D], torch.einsum("kr,hdr->khd", c, wk))
        s = (s + torch.einsum("qhd,kd->hqk", q[r0:r1, :, D:], kr)) * lw.scale
        p = torch.softmax(s.masked_fill(~see, float("-inf")), dim=-1)
        out[r0:r1] = torch.einsum("hqk,khv->qhv", p, torch.einsum("kr,hvr->khv", c, wv))
    if head_gate is not None:
        out = out * torch.sigmoid(head_gate.float())[..., None]
    o = out.reshape(T, H * V)
    if gate is not None:
        o = o * torch.sigmoid(gate.float())
    return o.to(pool.dtype)
