"""Grouped-query attention of listed layers: any head widths; optionally biases, per-head query / key norms, rotary positions on part
of a head (interleaved pairs or halves), a chunk mask (a query sees the keys of its own chunk of positions) or a sliding window that may
keep the first tokens of the sequence, soft-capped scores, a sink per head, a sigmoid gate per element or per head; sigmoid weights (with a
number per head added to the score) in place of the softmax; values that are cached rotated, their sums turned back by the query's
position.

One launch normalises, rotates and writes the new keys and values to their cache slots (``csrc/stream32.cu``).  Rows are then attended
in one of two ways, chosen per request of a batch:

* decoded tokens and short portions: every row is its own request of the decode kernel (``csrc/attn_grouped.cu``: page tiles on the
  tensor core, split over pages, gate in the combine);
* prompt chunks: the prefill kernel reads the pages themselves (``csrc/attn_window.cu``), gate in its epilogue.

float32 models and widths outside the tiling run every row through ``csrc/full32.cu``.  CPU tensors evaluate the PyTorch definition.
"""
from __future__ import annotations

import ctypes

import torch

from . import _lib
from . import latent as LA
from . import stream32 as S
from .attention import ROPE_INTERLEAVED, ROPE_NEOX, apply_rope_ref
from .basic import _ptr, _stream, dtype_code

P, I, F, LL = ctypes.c_void_p, ctypes.c_int, ctypes.c_float, ctypes.c_longlong
_lib.register_sigs({
    "fb_head_norm_rope": [P, LL, P, P, I, I, I, I, I, I, I, I, I, I, P, P, I, P, P, I, P, P, I, I, P, P, F, I, P],
    "fb_grouped_plan": [P, I, I, I, I, P, P, I, P],
    "fb_grouped_decode": [P, LL, P, P, P, LL, P, LL, P, P, P, P, P, P, I, I, I, I, I, LL, I, I, I, I, I, I, F, F, P, P, LL, P, P, P, I, I, I, P],
    "fb_grouped_attn32": [P, LL, P, P, P, LL, P, LL, P, P, I, I, I, I, I, I, I, I, I, I, I, I, F, F, P, P, LL, P, P, P, I, I, I, P],
    "fb_attn_window_paged": [P, LL, I, P, P, LL, P, I, P, LL, P, LL, P, I, I, I, I, I, I, I, I, F, F, P, P, LL, P, P, P, I, I, I, P],
}, ["attn_grouped"])

ROW_TOKENS = 16                  # requests that bring at most this many tokens take the decode kernel, a row each
_MAX_ROWS = 512                  # rows per call of the decode kernel


class GroupedWeights:
    """One attention layer.  ``dim`` / ``vdim`` are the true head widths, ``dp`` / ``vp`` the stored ones (multiples of 8; the padding is
    zero in the projections and in the cache)."""

    def __init__(self):
        self.heads = self.kv_heads = self.dim = self.vdim = self.dp = self.vp = 0
        self.window = self.keep = self.chunk = self.rot = 0
        self.rope_mode = ROPE_INTERLEAVED
        self.scale = 1.0
        self.softcap = 0.0
        self.own_kv = True       # False: keys and values come from another layer's cache
        self.gate = "elem"       # "elem": columns of the projection; "head": fp32 logits handed to ``attention``; "": none
        self.in_proj = None      # rows [queries | elementwise gate | keys | values]
        self.in_bias = None      # its bias, where the layer has one
        self.q_norm = self.k_norm = None
        self.unit_norm = False   # the per-head norm has no weights
        self.sinks = None        # fp32 [heads]
        self.score_bias = None   # fp32 [heads]: weights sigmoid(score + score_bias), not normalised
        self.rot_v = 0           # dimensions of a value that turn, stored as pairs (2m, 2m + 1)
        self.turn = None         # (cos, sin) tables of the values' rotation; the model sets them
        self.more_col = 0        # first of the further rows of the projection

    @property
    def gate_col(self) -> int:
        return self.heads * self.dp

    @property
    def k_col(self) -> int:
        return self.gate_col + (self.heads * self.vp if self.gate == "elem" else 0)

    @property
    def v_col(self) -> int:
        return self.k_col + self.kv_heads * self.dp


def value_order(spec):
    """Order in which a head's value dimensions are stored: the two of a rotated pair side by side (None: as they come)."""
    if not spec.rope_values or spec.rope_values.get("mode") != "neox":
        return None
    n = spec.rope_values["rot_dim"]
    pairs = torch.arange(n).view(2, n // 2).t().reshape(-1)
    return torch.cat([pairs, torch.arange(n, spec.vdim)])


def out_proj(o, spec):
    """Output projection [width, heads * vdim] with its columns in the stored order, zero columns where the heads are padded."""
    order = value_order(spec)
    if order is not None:
        o = o.reshape(o.shape[0], spec.heads, spec.vdim)[:, :, order.to(o.device)].reshape(o.shape[0], -1)
    return LA.pad_out_proj(o, spec)


def build(spec, q, k, v, g, q_norm, k_norm, biases=None, sinks=None, score_bias=None, more=()):
    """(GroupedWeights without ``in_proj``, merged input projection matrix) from the layer's matrices; ``k`` None: no own keys; ``g``
    None: no elementwise gate; ``biases``: those of q, k and v; ``more``: matrices that read the same input."""
    w = GroupedWeights()
    w.heads, w.kv_heads, w.dim, w.vdim = spec.heads, spec.kv_heads, spec.dim, spec.vdim
    w.dp, w.vp = LA._round8(spec.dim), LA._round8(spec.vdim)
    w.chunk, w.scale, w.own_kv = int(spec.chunk or 0), float(spec.scale), k is not None
    w.window, w.keep, w.softcap, w.gate = int(spec.window or 0), int(spec.keep or 0) if spec.window else 0, float(spec.softcap or 0.0), spec.gate
    w.rot = int(spec.rope["rot_dim"]) if spec.rope else 0
    w.rope_mode = ROPE_NEOX if spec.rope and spec.rope.get("mode") == "neox" else ROPE_INTERLEAVED
    w.q_norm, w.k_norm, w.unit_norm = q_norm, k_norm, bool(spec.qk_norm and not spec.norm_weight)
    w.sinks = sinks.float().contiguous() if sinks is not None else None
    w.score_bias = score_bias.float().contiguous() if spec.weights == "sigmoid" else None
    w.rot_v = int(spec.rope_values["rot_dim"]) if spec.rope_values else 0
    order = value_order(spec)

    def merge(q, g, k, v, more=()):
        parts = [LA._pad_heads(q, w.heads, w.dp)] + ([LA._pad_heads(g, w.heads, w.vp)] if g is not None else [])
        if k is not None:
            if order is not None:
                v = v.reshape(w.kv_heads, w.vdim, v.shape[1])[:, order.to(v.device)].reshape(v.shape)
            parts += [LA._pad_heads(k, w.kv_heads, w.dp), LA._pad_heads(v, w.kv_heads, w.vp)]
        w.more_col = sum(m.shape[0] for m in parts)
        return LA.pad_rows(torch.cat([*parts, *more], dim=0), 32)

    if biases is not None:
        bq, bk, bv = (b[:, None] if b is not None else None for b in biases)
        w.in_bias = merge(bq, bq.new_zeros((w.heads * w.vp, 1)) if g is not None else None, bk, bv)[:, 0].contiguous()
    return w, merge(q, g, k, v, more)


def first_key(pos, window: int, chunk: int):
    """First position of the chunk or window of a query at ``pos`` (tensors or integers)."""
    if chunk:
        return pos - pos % chunk
    if window:
        return (pos - window + 1).clamp(min=0) if torch.is_tensor(pos) else max(0, pos - window + 1)
    return pos * 0


def post(w: GroupedWeights, proj, fb, kv, cos, sin, eps: float) -> None:
    """Norm and rotation, where the layer has them, of the queries and keys in ``proj`` (in place; fp32 arithmetic) and the new keys and
    (rotated) values into their cache slots (rows with a negative slot are not cached)."""
    T = proj.shape[0]
    k_pool, v_pool = kv
    if proj.is_cuda:
        G = w.kv_heads if w.own_kv else 0
        cv, sv = w.turn if w.rot_v else (None, None)
        tab = cos if cos is not None else cv
        rc = _lib.kernels().fb_head_norm_rope(_ptr(proj), proj.stride(0), _ptr(fb.positions), _ptr(fb.slots), T, w.heads, G, w.dim, w.dp, w.vp, w.k_col,
                                              w.v_col, w.rot, 1 if w.rope_mode == ROPE_NEOX else 0, _ptr(w.q_norm), _ptr(w.k_norm), int(w.unit_norm), _ptr(cos), _ptr(sin), w.rot_v,
                                              _ptr(cv), _ptr(sv), tab.shape[0] if tab is not None else 0,
                                              k_pool.shape[0] * k_pool.shape[1], _ptr(k_pool), _ptr(v_pool), float(eps), S.act_code(proj.dtype), _stream())
        _lib.check(rc, "fb_head_norm_rope")
        return

    def turn(col, heads, norm_w):
        x = proj[:, col:col + heads * w.dp].reshape(T, heads, w.dp).clone()
        if norm_w is not None or w.unit_norm:
            x[..., :w.dim] = S._rms(x[..., :w.dim].float(), norm_w if norm_w is not None else torch.ones(()), eps).to(x.dtype)
        return apply_rope_ref(x, fb.positions, cos, sin, w.rope_mode, w.rot) if w.rot else x

    proj[:, :w.gate_col] = turn(0, w.heads, w.q_norm).reshape(T, -1)
    if w.own_kv:
        ok = fb.slots >= 0
        sl = fb.slots[ok].long()
        k_pool.view(-1, w.kv_heads, w.dp)[sl] = turn(w.k_col, w.kv_heads, w.k_norm)[ok].to(k_pool.dtype)
        v = proj[:, w.v_col:w.v_col + w.kv_heads * w.vp].reshape(T, w.kv_heads, w.vp)
        if w.rot_v:
            v = apply_rope_ref(v, fb.positions, *w.turn, ROPE_INTERLEAVED, w.rot_v)
        v_pool.view(-1, w.kv_heads, w.vp)[sl] = v[ok].to(v_pool.dtype)


# ---------------------------------------------------------------------------------------------------
# batch plans, shared by all such layers of a forward pass
# ---------------------------------------------------------------------------------------------------
class GroupedPlan:
    def __init__(self):
        self.rows = None             # int64 rows of the packed batch that are their own requests (None: all of them)
        self.n_rows = 0
        self.page_table = None       # [n_rows, P] and [n_rows]
        self.kv_lens = None
        self.blocks = None           # prefill query blocks: (packed row, position, rows, 0, 0, request)
        self.n_blocks = 0
        self.lists: dict = {}        # (window, keep, chunk, first row) -> work list of the decode kernel


def build_plan(fb, prefill: bool) -> GroupedPlan:
    pl = GroupedPlan()
    if fb.is_decode:
        pl.page_table, pl.kv_lens, pl.n_rows = fb.page_table, fb.kv_lens, fb.page_table.shape[0]
        return pl
    dev = fb.page_table.device
    cu = fb.cu_q_host if fb.cu_q_host is not None else fb.cu_q.tolist()
    lens = fb.kv_lens_host if fb.kv_lens_host is not None else fb.kv_lens.tolist()
    reqs = [b for b in range(len(cu) - 1) if cu[b + 1] > cu[b]]
    long = [b for b in reqs if prefill and cu[b + 1] - cu[b] > ROW_TOKENS]
    short = [b for b in reqs if b not in set(long)]
    if short:
        owner, rows = LA._row_plan(fb, short, cu, dev)
        pl.n_rows = rows.shape[0]
        pl.page_table = fb.page_table.index_select(0, owner)
        seen = (fb.positions + 1).to(torch.int32)
        pl.kv_lens = seen.index_select(0, rows) if long else seen
        pl.rows = rows if long else None
    blocks = []
    for b in long:
        n = cu[b + 1] - cu[b]
        blocks += [(cu[b] + q0, lens[b] - n + q0, min(256, n - q0), 0, 0, b) for q0 in range(0, n, 256)]
    if blocks:
        blocks.sort(key=lambda t: -t[1])                                    # most keys first (unmasked layers)
        pl.blocks, pl.n_blocks = torch.tensor(blocks, dtype=torch.int32).to(dev, non_blocking=True), len(blocks)
    return pl


def _plan(fb, prefill: bool) -> GroupedPlan:
    cache = fb.__dict__.setdefault("_grouped_plans", {})
    if prefill not in cache:
        cache[prefill] = build_plan(fb, prefill)
    return cache[prefill]


def decode_ok(w, dtype, page_len: int) -> bool:
    return dtype in (torch.float16, torch.bfloat16) and w.dp <= 256 and w.vp <= 256 and page_len == 128


def prefill_ok(w, dtype, page_len: int) -> bool:
    if dtype not in (torch.float16, torch.bfloat16) or page_len != 128:
        return False
    ok = w.__dict__.get("_prefill_ok")
    if ok is None:
        ok = w._prefill_ok = bool(_lib.kernels()._lib.fb_attn_window_supported(w.dp, 0, w.vp))
    return ok


def _splits(w, max_pages: int, page_len: int) -> int:
    """Most pages one query's visible keys touch."""
    span = w.chunk or w.window
    return min(max_pages, (span + page_len - 2) // page_len + 1 + (w.keep + page_len - 1) // page_len) if span else max_pages


_SCRATCH: dict = {}


def _scratch(dev, n: int, kind: str):
    """fp32 scratch of at least ``n`` elements, shared by the layers of a model (they run one after another)."""
    if torch.cuda.is_current_stream_capturing():
        return torch.empty((n,), device=dev, dtype=torch.float32)           # owned by the graph
    t = _SCRATCH.get((dev, kind))
    if t is None or t.numel() < n:
        t = _SCRATCH[(dev, kind)] = torch.empty((n,), device=dev, dtype=torch.float32)
    return t


def _gate_args(gate):
    return _ptr(gate), gate.stride(0) if gate is not None else 0


def _weight_args(w):
    """Sigmoid weights and the rotation of the outputs."""
    cv, sv = w.turn if w.rot_v else (None, None)
    return _ptr(w.score_bias), _ptr(cv), _ptr(sv), w.rot_v, cv.shape[0] if cv is not None else 0


def decode_rows(w, pl: GroupedPlan, q, gate, head_gate, kv, page_table, kv_lens, out, row0: int = 0) -> None:
    """Rows ``q`` [n, heads * dp] against their own page-table rows; gated heads to ``out`` [n, heads * vp] (row strides free).  ``gate``
    [n, heads * vp] and ``head_gate`` (fp32 [n, heads]): None where the layer has no such gate."""
    k_pool, v_pool = kv
    n, page_len, max_pages, lib = q.shape[0], k_pool.shape[1], page_table.shape[1], _lib.kernels()
    slots = k_pool.shape[0] * page_len
    if not decode_ok(w, q.dtype, page_len):
        rc = lib.fb_grouped_attn32(_ptr(q), q.stride(0), _ptr(k_pool), _ptr(v_pool), _ptr(out), out.stride(0), *_gate_args(gate),
                                   _ptr(page_table), _ptr(kv_lens), n, w.heads, w.kv_heads, w.dim, w.dp, w.vp, page_table.stride(0), k_pool.shape[0],
                                   page_len, w.window, w.chunk, w.keep, w.scale, w.softcap, _ptr(w.sinks), *_gate_args(head_gate), *_weight_args(w),
                                   S.act_code(q.dtype), _stream())
        _lib.check(rc, "fb_grouped_attn32")
        return
    if n > _MAX_ROWS:
        for i in range(0, n, _MAX_ROWS):
            s = slice(i, i + _MAX_ROWS)
            decode_rows(w, pl, q[s], gate[s] if gate is not None else None, head_gate[s] if head_gate is not None else None, kv, page_table[s],
                        kv_lens[s], out[s], row0 + i)
        return
    splits = _splits(w, max_pages, page_len)
    key = (w.window, w.keep, w.chunk, row0)
    lst = pl.lists.get(key)
    if lst is None:
        lst = pl.lists[key] = torch.empty((2 * n * splits + 1,), device=q.device, dtype=torch.int32)
        _lib.check(lib.fb_grouped_plan(_ptr(kv_lens), n, w.window, w.chunk, w.keep, _ptr(lst[1:]), _ptr(lst), n * splits, _stream()), "fb_grouped_plan")
    part_o, part_ml = _scratch(q.device, n * w.heads * splits * w.vp, "o"), _scratch(q.device, n * w.heads * splits * 2, "ml")
    rc = lib.fb_grouped_decode(_ptr(q), q.stride(0), _ptr(k_pool), _ptr(v_pool), _ptr(out), out.stride(0), *_gate_args(gate), _ptr(page_table),
                               _ptr(kv_lens), _ptr(lst[1:]), _ptr(lst), _ptr(part_o), _ptr(part_ml), n, w.heads, w.kv_heads, w.dp, w.vp, slots,
                               page_table.stride(0), splits, n * splits, w.window, w.chunk, w.keep, w.scale, w.softcap, _ptr(w.sinks), *_gate_args(head_gate),
                               *_weight_args(w), dtype_code(q.dtype), _stream())
    _lib.check(rc, "fb_grouped_decode")


def prefill_blocks(w, pl: GroupedPlan, q, gate, head_gate, kv, page_table, out) -> None:
    k_pool, v_pool = kv
    rc = _lib.kernels().fb_attn_window_paged(_ptr(q), q.stride(0), q.shape[0], _ptr(k_pool), _ptr(v_pool), k_pool.shape[0] * k_pool.shape[1],
                                             _ptr(page_table), page_table.stride(0), _ptr(out), out.stride(0), *_gate_args(gate), _ptr(pl.blocks),
                                             pl.n_blocks, w.heads, w.kv_heads, w.dp, w.vp, w.window, w.chunk, w.keep, w.scale, w.softcap, _ptr(w.sinks),
                                             *_gate_args(head_gate), *_weight_args(w), dtype_code(q.dtype), _stream())
    _lib.check(rc, "fb_attn_window_paged")


def attention(w: GroupedWeights, proj, kv, fb, out=None, head_gate=None):
    """``proj`` after ``post`` (the new keys and values are cached already) -> gated heads ``[T, heads * vp]`` (``out``, where given).
    ``head_gate``: fp32 logits [T, heads] of a layer with one gate per head."""
    T = proj.shape[0]
    q, gate = proj[:, :w.gate_col], proj[:, w.gate_col:w.k_col] if w.gate == "elem" else None
    if not proj.is_cuda:
        y = attention_ref(w, q, gate, kv, fb, head_gate)
        return y if out is None else out.copy_(y)
    if out is None:
        out = torch.empty((T, w.heads * w.vp), device=proj.device, dtype=proj.dtype)
    pl = _plan(fb, prefill_ok(w, proj.dtype, kv[0].shape[1]) and not fb.is_decode)
    if pl.n_rows and pl.rows is None:
        decode_rows(w, pl, q, gate, head_gate, kv, pl.page_table, pl.kv_lens, out)
    elif pl.n_rows:
        part = torch.empty((pl.n_rows, w.heads * w.vp), device=proj.device, dtype=proj.dtype)
        sub = proj[:, :w.k_col].index_select(0, pl.rows)
        decode_rows(w, pl, sub[:, :w.gate_col], sub[:, w.gate_col:] if gate is not None else None,
                    head_gate.index_select(0, pl.rows) if head_gate is not None else None, kv, pl.page_table, pl.kv_lens, part)
    if pl.n_blocks:
        prefill_blocks(w, pl, q, gate, head_gate, kv, fb.page_table, out)
    if pl.n_rows and pl.rows is not None:
        out.index_copy_(0, pl.rows, part)
    return out


def attention_ref(w, q, gate, kv, fb, head_gate=None):
    """PyTorch evaluation over the pages (CPU tensors)."""
    T, H, G = q.shape[0], w.heads, w.kv_heads
    k_pool, v_pool = kv
    page_len = k_pool.shape[1]
    cu = fb.cu_q_host if fb.cu_q_host is not None else fb.cu_q.tolist()
    out = torch.zeros((T, H, w.vp), dtype=torch.float32)
    for b, L in enumerate(fb.kv_lens.tolist()):
        r0, r1 = cu[b], cu[b + 1]
        if r1 == r0 or L == 0:
            continue
        pages = fb.page_table[b, :(L + page_len - 1) // page_len].long()
        k = k_pool[pages].reshape(-1, G, w.dp)[:L].float().repeat_interleave(H // G, dim=1)
        v = v_pool[pages].reshape(-1, G, w.vp)[:L].float().repeat_interleave(H // G, dim=1)
        qpos, kpos = torch.arange(L - (r1 - r0), L)[:, None], torch.arange(L)[None, :]
        see = (kpos <= qpos) & ((kpos >= first_key(qpos, w.window, w.chunk)) | (kpos < w.keep))
        s = torch.einsum("qhd,khd->hqk", q[r0:r1].float().reshape(-1, H, w.dp), k) * w.scale
        if w.softcap:
            s = torch.tanh(s / w.softcap) * w.softcap
        if w.score_bias is not None:
            out[r0:r1] = torch.einsum("hqk,khv->qhv", torch.sigmoid(s + w.score_bias[:, None, None]) * see, v)
            continue
        s = s.masked_fill(~see, float("-inf"))
        if w.sinks is not None:
            s = torch.cat([s, w.sinks.view(H, 1, 1).expand(-1, s.shape[1], 1)], dim=-1)
        out[r0:r1] = torch.einsum("hqk,khv->qhv", torch.softmax(s, dim=-1)[..., :L], v)
    if w.rot_v:
        cv, sv = w.turn
        out = apply_rope_ref(out, fb.positions, cv, -sv, ROPE_INTERLEAVED, w.rot_v)
    if head_gate is not None:
        out = out * torch.sigmoid(head_gate.float())[..., None]
    out = out.reshape(T, -1)
    return (out * torch.sigmoid(gate.float()) if gate is not None else out).to(q.dtype)
