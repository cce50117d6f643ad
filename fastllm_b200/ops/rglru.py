"""Real-gated linear recurrent unit (the recurrent block of Griffin): one fp32 state per channel and request.

    u = conv(x),  r, i = sigmoid of two block-diagonal products of u
    log a = -8 r softplus(lam) ,  S <- a S + sqrt(1 - a^2) i u ,  out = S * gelu(y)

``x`` and ``y`` are two projections of the layer's input, ``conv`` a short causal convolution per channel whose last inputs belong to the
request's state.  Both live in the engine's state slots: ``[width, taps - 1]`` inputs in the activation type and ``[width]`` in fp32.

Three steps on CUDA (``csrc/rglru.cu``): the convolution, the gates' logits as one block-diagonal tensor-core product with fp32 results
(``basic.linear_blocks``), and the recurrence with the output gate: token by token for short portions, in chunks of 128 tokens that run
in parallel behind a launch that sums every chunk up for longer ones.  CPU tensors evaluate the PyTorch definition.
"""
from __future__ import annotations

import ctypes

import torch
import torch.nn.functional as F

from . import _lib
from . import basic as B
from . import latent as LA
from . import stream32 as S
from .basic import _ptr, _stream

P, I, LL = ctypes.c_void_p, ctypes.c_int, ctypes.c_longlong
_lib.register_sigs({
    "fb_rglru": [I, P, P, LL, P, P, P, P, P, P, P, LL, P, P, P, P, I, I, I, P, P, P, I, I, I, I, P],
}, ["rglru"])

CHUNK = 128
ROW_TOKENS = 16                  # requests that bring at most this many tokens walk them one by one
DECAY = 8.0                      # log a = -DECAY * r * softplus(lam)


class RGLRUWeights:
    """``width`` is the stored width: every block's channels padded to ``part`` (a multiple of 8); a padded channel's input, gate and output
    rows are zero, so its state stays zero."""

    def __init__(self):
        self.width = self.blocks = self.part = self.taps = 0
        self.in_proj = None      # rows [y | x | the layer's further rows]
        self.conv_w = None       # fp32 [taps, width]
        self.conv_b = None       # fp32 [width]
        self.gates = None        # [blocks, 2 * part, part]: rows of r, then of i
        self.gate_b = None       # fp32 [blocks, 2, part]
        self.decay = None        # fp32 [width]: -DECAY * softplus(lam)
        self.more_col = 0        # first of the further rows


def stored_width(spec) -> int:
    return spec.blocks * LA._round8(spec.width // spec.blocks)


def build(spec, y, x, conv_w, conv_b, ra, ra_b, ri, ri_b, lam, more=()):
    """(RGLRUWeights without ``in_proj``, merged input projection matrix) from the layer's tensors; ``more``: matrices that read the same
    input."""
    w = RGLRUWeights()
    n = spec.width // spec.blocks
    w.blocks, w.part, w.taps, w.width = spec.blocks, LA._round8(n), conv_w.shape[1], stored_width(spec)
    rows = lambda m: LA._pad_heads(m, w.blocks, w.part)
    vec = lambda v: rows(v.reshape(-1, 1))[:, 0].float().contiguous()
    w.conv_w, w.conv_b = rows(conv_w).float().t().contiguous(), vec(conv_b)
    square = lambda m: F.pad(m, (0, w.part - n, 0, w.part - n))
    w.gates = torch.cat([square(ra), square(ri)], dim=1).contiguous()
    w.gate_b = torch.stack([vec(ra_b).view(w.blocks, w.part), vec(ri_b).view(w.blocks, w.part)], dim=1).contiguous()
    w.decay = vec(-DECAY * F.softplus(lam.double()))
    w.more_col = 2 * w.width
    return w, LA.pad_rows(torch.cat([rows(y), rows(x), *more], dim=0), 32)


def in_bias(w, y_b, x_b, more, rows: int):
    """The merged projection's bias, ``rows`` long; ``more``: biases of the further rows."""
    pad = lambda b: LA._pad_heads(b[:, None], w.blocks, w.part)[:, 0]
    b = torch.cat([pad(y_b), pad(x_b), *more])
    return F.pad(b, (0, rows - b.shape[0])).contiguous()


def out_proj(o, spec):
    """Output projection [H, width] with zero columns where the blocks are padded."""
    return LA._pad_heads(o.t().contiguous(), spec.blocks, LA._round8(spec.width // spec.blocks)).t().contiguous()


class _Plan:
    """The batch's requests: ``conv`` all of them in chunks, ``short`` those that are walked token by token, ``long`` the others in chunks.  Items are
    (first row, rows, slot, the request's rows before it, its first item in the list, last)."""

    def __init__(self, fb):
        cu, lists = fb.cu_q_host, ([], [], [])
        for b, s in enumerate(fb.state_slots_host):
            n = cu[b + 1] - cu[b]
            for l in (lists[0], lists[2])[:1 if n <= ROW_TOKENS else 2]:
                first = len(l)
                l.extend((cu[b] + c, min(CHUNK, n - c), s, c, first, int(c + CHUNK >= n)) for c in range(0, n, CHUNK))
            if 0 < n <= ROW_TOKENS:
                lists[1].append((cu[b], n, s, 0, 0, 1))
        self.max_rows = max((c[1] for c in lists[0]), default=1)
        self.multi = any(not c[5] for c in lists[2])
        self.sizes = [len(l) for l in lists]
        meta = torch.tensor([x for l in lists for t in l for x in t], dtype=torch.int32).to(fb.page_table.device, non_blocking=True)
        self.conv, self.short, self.long = meta.split([6 * n for n in self.sizes])


def mix(w: RGLRUWeights, proj, fb, state):
    """``proj`` [T, >= y and x] -> gated states [T, width]; advances ``state`` ([slots, width, taps - 1], fp32 [slots, width]) of every request of
    the batch."""
    if not proj.is_cuda:
        return mix_ref(w, proj, fb, state)
    T, W = proj.shape[0], w.width
    u = torch.empty((T, W), device=proj.device, dtype=proj.dtype)
    out = torch.empty_like(u)

    def step(which, z, slots, items, n, rows=1, sums=None):
        rc = _lib.kernels().fb_rglru(which, _ptr(proj[:, W:]), _ptr(proj), proj.stride(0), _ptr(w.conv_w), _ptr(w.conv_b), _ptr(w.gate_b), _ptr(w.decay), _ptr(z), _ptr(u),
                                     _ptr(out), out.stride(0), _ptr(state[0]), _ptr(state[1]), _ptr(slots), _ptr(items), n, rows, int(sums is not None),
                                     *(_ptr(t) for t in (sums if sums is not None else (None,) * 3)), W, w.part, w.taps, S.act_code(proj.dtype), _stream())
        _lib.check(rc, "fb_rglru")

    if fb.is_decode:
        step(0, None, fb.state_slots, None, T)
        step(1, B.linear_blocks(u, w.gates), fb.state_slots, None, T)
        return out
    pl = fb.__dict__.get("_rglru_plan")
    if pl is None:
        pl = fb._rglru_plan = _Plan(fb)
    n_conv, n_short, n_long = pl.sizes
    step(0, None, None, pl.conv, n_conv, pl.max_rows)
    z = B.linear_blocks(u, w.gates)
    step(1, z, None, pl.short, n_short)
    step(2, z, None, pl.long, n_long, pl.max_rows, torch.empty((3, n_long, W), device=proj.device, dtype=torch.float32) if pl.multi else None)
    return out


def mix_ref(w: RGLRUWeights, proj, fb, state):
    """PyTorch evaluation, token by token (CPU tensors)."""
    W, K = w.width, w.taps
    y, x = F.gelu(proj[:, :W].float(), approximate="tanh"), proj[:, W:2 * W]
    out = torch.empty((proj.shape[0], W), dtype=torch.float32)
    cu = fb.cu_q_host if fb.cu_q_host is not None else fb.cu_q.tolist()
    for b, slot in enumerate(fb.state_slots.tolist()):
        r0, r1 = cu[b], cu[b + 1]
        seq = torch.cat([state[0][slot].t(), x[r0:r1]])                     # [K - 1 + n, W]
        u = sum(seq[k:k + r1 - r0].float() * w.conv_w[k] for k in range(K)) + w.conv_b
        u = u.to(proj.dtype)
        z = (B.linear_blocks(u, w.gates).view(-1, w.blocks, 2, w.part) + w.gate_b).sigmoid()
        r, i = z[:, :, 0].reshape(-1, W), z[:, :, 1].reshape(-1, W)
        log_a = r * w.decay
        a, add = log_a.exp(), (-torch.expm1(2 * log_a)).sqrt() * i * u.float()
        St = state[1][slot]
        for t in range(r1 - r0):
            St.mul_(a[t]).add_(add[t])
            out[r0 + t] = St
        state[0][slot] = seq[seq.shape[0] - (K - 1):].t()
    return (out * y).to(proj.dtype)
