"""Vuripel (attention with sinks and soft caps, windowed attention that keeps the first tokens, matrix-memory LSTM, parallel blocks with
grouped softmax routing, looped passes, per-layer token inputs) against its plain statement.

Every case builds a small random model of its own.  The CPU runs use the framework's PyTorch operator definitions (scheduling,
cache, loading and the model itself); the GPU runs the kernels, in float32 and bfloat16.
"""
import json

import pytest
import torch

from . import listed_common as LC
from . import vuripel_oracle as O
from .listed_common import DEVICES, PAGE, assert_close, few_threads, portions, save  # noqa: F401
from fastllm_b200.engine import EngineConfig, GenerationConfig, LLMEngine
from fastllm_b200.engine.replay import Replay, open_engine
from fastllm_b200.loader.hf import load_model
from fastllm_b200.models.config import AttnSpec, MLSTMSpec, from_hf_dict
from fastllm_b200.models.decoder import ForwardBatch
from fastllm_b200.ops import attention as A
from fastllm_b200.ops import basic as B
from fastllm_b200.ops import grouped as GR
from fastllm_b200.ops import mlstm as ML
from fastllm_b200.ops import moe as MOE
from fastllm_b200.ops import stream32 as S
from fastllm_b200.ops.quant import LinearWeight

gpu = pytest.mark.gpu


def full(heads, kv, dim, vdim, cap=12.0, scale=None):
    return "attention", {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or 0.9 * dim ** -0.5, "softcap": cap}


def local(heads, kv, dim, vdim, size, keep, rot, cap=9.0, scale=None, base=1e4):
    return "attention_2", {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or 0.7 * dim ** -0.5, "softcap": cap,
                           "mask": {"size": size, "keep_first": keep}, "rot": {"base": base, "dims": rot}}


def cell(heads, dim, vdim, cap=7.0):
    return "mlstm", {"heads": heads, "dim": dim, "vdim": vdim, "gate_cap": cap}


def dense(ff):
    return {"kind": "dense", "ff": ff}


def moe(experts, top, ff, shared=None, groups=None):
    out = {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}}
    if shared:
        out["shared"] = {"ff": shared}
    if groups:
        out["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    return out


def config(layers, width=160, vocab=304, eps=1e-5, loop=None, side=None):
    cfg = {"architecture": "Vuripel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}
    if loop:
        cfg["loop"] = dict(zip(("start", "stop", "times"), loop))
    if side:
        cfg["token_side"] = {"dim": side}
    return cfg


CONFIGS = {
    # every expert is taken (no close calls in 16 bits); a loop in the middle, two windows, a layer without feed-forward
    "mixed": config([(local(6, 3, 40, 24, 50, 5, 16), moe(3, 3, 48, 72)), (cell(3, 24, 40), None), (full(6, 2, 40, 24), dense(200)),
                     (cell(2, 64, 16), moe(2, 2, 112)), (local(4, 4, 64, 72, 150, 131, 64), dense(64))], loop=(1, 3, 3), side=24),
    # nothing is a multiple of anything the kernels tile; the loop opens the stack
    "odd": config([(cell(3, 20, 12), moe(3, 3, 75, 30)), (local(3, 1, 20, 12, 19, 1, 6, scale=0.3), dense(75)), (full(3, 3, 20, 12, scale=0.2), None),
                   (cell(1, 33, 50), dense(31))], width=148, vocab=331, eps=1e-4, loop=(0, 2, 2), side=10),
    # heads of a served size: sixteen query heads per key head, whole tensor-core tiles, wide states
    "wide": config([(full(32, 2, 128, 128, cap=40.0), moe(2, 2, 128, 256)), (cell(4, 128, 128), moe(4, 4, 64)), (local(32, 2, 128, 128, 200, 16, 64), dense(512)),
                    (cell(2, 64, 192), None), (local(24, 1, 192, 256, 130, 129, 192), None)], width=256, vocab=512, loop=(4, 5, 2), side=64),
    # one of everything; a window of one token, one kept token, a single pass
    "ones": config([(full(1, 1, 8, 8), moe(1, 1, 8, 8, (1, 1))), (local(1, 1, 8, 8, 1, 1, 8), dense(8)), (cell(1, 16, 24), moe(1, 1, 8))], width=64, vocab=64,
                   loop=(0, 3, 1), side=1),
    # none of the optional parts
    "bare": config([(cell(2, 32, 32), None), (full(4, 2, 32, 32), moe(2, 2, 40)), (local(4, 1, 32, 32, 33, 0, 32), None)], width=128, vocab=200),
    # experts are chosen within their best groups
    "routed": config([(full(4, 2, 32, 32), moe(40, 3, 64, 96, (8, 3))), (cell(2, 32, 32), moe(6, 1, 40, None, (3, 1)))], width=128, vocab=256, side=16),
}
OVER = {"routed": 0.5, "ones": 0.15}      # "ones": a single head that nearly cancels before its norm has no other beside it
_CACHE: dict = {}


def weights(name):
    if name not in _CACHE:
        _CACHE[name] = O.random_weights(CONFIGS[name], seed=len(name))
    return _CACHE[name]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, weights, checkpoint folder); the folders are written once."""
    root, out = tmp_path_factory.mktemp("vuripel"), {}

    def get(name):
        if name not in out:
            out[name] = (CONFIGS[name], weights(name), save(root / name, CONFIGS[name], weights(name)))
        return out[name]
    return get


def oracle(name, tokens):
    key = (name, tuple(tokens))
    if key not in _CACHE:
        _CACHE[key] = O.forward(CONFIGS[name], weights(name), tokens)
    return _CACHE[key]


def prompt(name, n, seed=0):
    g = torch.Generator().manual_seed(1000 * seed + n)
    return torch.randint(0, CONFIGS[name]["vocab"], (n,), generator=g).tolist()


def replay(models, name, where, reqs, schedule, max_tokens):
    LC.replay(models(name)[2], where, reqs, schedule, max_tokens, lambda toks: oracle(name, toks), OVER.get(name, 0.01), 0.05)


# ---------------------------------------------------------------------------------------------------
# the model through cache, state and batches
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts(models, name, where):
    reqs = {str(n): prompt(name, n) for n in ((1, 2, 17, 130, 300) if where[0] == "cuda" else (1, 2, 17, 130))}
    replay(models, name, where, reqs, [[(r, len(t))] for r, t in reqs.items()], 384)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_token_by_token(models, name, where):
    """From the first token on, across page borders, past every window that is shorter and its kept tokens."""
    n = 40 if where[0] == "cpu" else 300
    replay(models, name, where, {"a": prompt(name, n, 1) if n != 300 else prompt(name, n)}, [[("a", 1)]] * n, 384)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("sizes", [(2,), (3, 16, 17), (64, 5), (127, 1, 2), (37, 129, 2, 1)], ids=str)
def test_portions(models, sizes, where):
    n = 130 if where[0] == "cpu" else 300
    for name in ("mixed", "odd", "wide") if where[0] == "cuda" else ("odd",):
        replay(models, name, where, {"a": prompt(name, n)}, [[("a", k)] for k in portions(n, sizes)], 384)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide", "routed"])
def test_unequal_requests_and_reused_slots(models, name, where):
    """Prompts of several requests next to decoded tokens of others, requests that pause, pages and state slots that change owner."""
    if where[0] == "cpu" and name in ("wide", "routed"):
        pytest.skip("the CPU runs the other two")
    reqs = {"a": prompt(name, 210, 3), "b": prompt(name, 33, 4), "c": prompt(name, 129, 5), "d": prompt(name, 3, 6), "e": prompt(name, 180, 7),
            "f": prompt(name, 140, 8)}
    sched = [[("a", 100), ("b", 30), ("c", 2), ("d", 1)], [("b", 1), ("a", 1), ("d", 1)], [("c", 60), ("d", 1), ("b", 1), ("a", 1)], [("b", 1)],
             [("a", 1), ("c", 1), ("e", 40)], [("a", 50), ("c", 60), ("e", 2)], [("a", 1), ("c", 1), ("e", 1)], [("c", 5), ("e", 100), ("a", 1)]]
    done = {}
    for step in sched:
        for r, n in step:
            done[r] = done.get(r, 0) + n
    sched.append([(r, len(reqs[r]) - done[r]) for r in ("a", "e") if len(reqs[r]) > done[r]])
    sched += [[("f", 130)]] + [[("f", 1)]] * 10
    assert all(done[r] == len(reqs[r]) for r in "bcd")
    # tight pool: "e" and "f" only fit because earlier requests gave their pages and slots back
    replay(models, name, where, reqs, sched, 6 * PAGE)


@pytest.mark.parametrize("where", DEVICES)
def test_batch_alone(models, where):
    """Each request of a batch computes what it computes alone, to rounding."""
    device, dtype = where
    path, reqs = models("mixed")[2], [prompt("mixed", n, 11) for n in (70, 1, 18, 33)]
    eng = open_engine(path, dtype, 8 * PAGE, device)
    rp = Replay(eng)
    last = lambda t: [len(t) - 1]
    both = rp.step([(str(i), t, last(t)) for i, t in enumerate(reqs)])
    more = rp.step([(str(i), [5 + i], [0]) for i in range(4)], [str(i) for i in range(4)])
    for i in (2, 0, 3, 1):
        a, b = rp.step([("x", reqs[i], last(reqs[i]))]), rp.step([("x", [5 + i], [0])], ["x"])
        assert_close(torch.cat([both[i:i + 1], more[i:i + 1]]), torch.cat([a, b]).double(), dtype, 0.03)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
def test_long_decoding(models, dtype):
    n = 420
    for name in ("mixed", "wide"):
        replay(models, name, ("cuda", dtype), {"a": prompt(name, n, 9)}, [[("a", 5)]] + [[("a", 1)]] * (n - 5), 512)


# ---------------------------------------------------------------------------------------------------
# window edges and kept tokens: with one attention layer, a token reaches exactly the rows that see it
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("size,keep", [(1, 0), (2, 1), (31, 4), (64, 64), (100, 130), (128, 1), (129, 3)], ids=str)
def test_who_sees_a_token(tmp_path, size, keep, where):
    device, dtype = where
    cfg = config([(local(2, 1, 32, 32, size, keep, 16), None)], width=64, vocab=96)
    w = O.random_weights(cfg, seed=size)
    path = save(tmp_path / "m", cfg, w)
    n = max(PAGE, keep) + 2 * size + 40
    g = torch.Generator().manual_seed(size)
    base = torch.randint(0, 96, (n,), generator=g).tolist()
    w64 = {k: v.double() for k, v in w.items()}
    ref = O.forward(cfg, w64, base)
    eng = open_engine(path, dtype, 512, device)

    def run(seq, cut):
        rp, at, rows = Replay(eng), 0, []
        for c in cut:
            rows.append(rp.step([("r", seq[at:at + c], list(range(c)))], ["r"] if at + c == n else []))
            at += c
        return torch.cat(rows)

    for p in sorted({0, keep - 1, keep, PAGE - 1, PAGE, n - size - 30} - {-1}):
        last = n - 1 if p < keep else min(n - 1, p + size - 1)          # the last row that sees position p
        # the substitute is the token that moves that row most
        cand = torch.randint(0, 96, (12,), generator=g).tolist()
        alts = {t: O.forward(cfg, w64, base[:p] + [t] + base[p + 1:]) for t in cand if t != base[p]}
        best = max(alts, key=lambda t: (alts[t] - ref)[last].abs().max().item())
        want = (alts[best] - ref).abs().amax(-1)
        assert want[:p].max() == 0 if p else True
        assert want[last] > 0 and (last == n - 1 or want[last + 1:].max() == 0)
        other = base[:p] + [best] + base[p + 1:]
        for cut in ([n], [p + size // 2 + 1, n - p - size // 2 - 1], [n - 20] + [1] * 20):
            if min(cut) <= 0 or (device == "cpu" and len(cut) > 2):
                continue
            diff = (run(base, cut) - run(other, cut)).abs().amax(-1)
            noise = 1e-5 if dtype == torch.float32 else 1e-6            # rows that do not see the token are computed alike, bit for bit
            assert (p == 0 or diff[:p].max() <= noise) and (last == n - 1 or diff[last + 1:].max() <= noise), "a row that must not see the token does"
            assert (diff[last] - want[last]).abs() < 0.05 * want[last] + (1e-4 if dtype == torch.float32 else 0.06), "the last row that sees the token misses it"


# ---------------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("width", [64, 148, 75])
def test_residual_and_pass_starts(width, where):
    """Embedding with a step vector; residual, step vector and repeated embedding in front of the next norm; with and without its parts."""
    device, dtype = where
    g = torch.Generator().manual_seed(width)
    r16 = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    table, vec, nw, pw, y = r16(50, width), r16(width), r16(width), r16(width), r16(6, width)
    ids, h0 = torch.randint(0, 50, (6,), generator=g), torch.randn(6, width, generator=g)
    to = lambda t: t.to(device, dtype)
    tol = 2e-5 if dtype == torch.float32 else 0.03
    tab, v, di = to(table), to(vec), ids.int().to(device)
    h, x = S.embed_pos_norm(di, di, tab, None, to(nw), 1e-5, add_vec=v)
    want = table[ids].double() + vec.double()
    assert (h.cpu().double() - want).abs().max() < 2e-6
    assert (x.cpu().double() - O.rms_norm(want, nw.double(), 1e-5)).abs().max() < tol * 8
    for start in (None, (None, di, v), (tab, di, v)):
        for post in (None, pw):
            for out in (y, None):
                if out is None and post is not None:
                    continue
                h = h0.clone().to(device)
                x = S.add_norm(h, to(out) if out is not None else None, to(post) if post is not None else None, to(nw), 1e-4, start=start)
                want = h0.double()
                if out is not None:
                    want = want + (O.rms_norm(out.double(), post.double(), 1e-4) if post is not None else out.double())
                if start is not None:
                    want = want + vec.double() + (table[ids].double() if start[0] is not None else 0)
                assert (h.cpu().double() - want).abs().max() < 2e-5
                ref = O.rms_norm(want, nw.double(), 1e-4)
                assert (x.cpu().double() - ref).abs().max() < tol * (1 + ref.abs().max())


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("shape", [(3, 64, 128), (300, 96, 72), (700, 256, 512), (5, 75, 33), (270, 40, 24)], ids=str)
def test_product_epilogues(shape, where):
    """GELU in both forms, a gate per row, rows of a table, gated GELU units, the residual with its copy."""
    device, dtype = where
    M, N, K = shape
    g = torch.Generator().manual_seed(N)
    r16 = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    x, w, table, rows, gate = r16(M, K), (r16(N, K) * 1.5 * K ** -0.5).to(torch.bfloat16), r16(20, N + 40), torch.randint(0, 20, (M,), generator=g), torch.randn(M, 3, generator=g)
    to = lambda t: t.to(device, dtype)
    lw = LinearWeight.from_dense(to(w), act_dtype=dtype)
    lw.exact32 = dtype == torch.float32
    z = O.linear(w.double(), x.double())
    ok = lambda got, want, tol16=0.02: (got.cpu().double() - want).abs().max() < (2e-5 if dtype == torch.float32 else tol16) * (1 + want.abs().max())
    gd, td = gate.to(device), to(table)
    assert ok(lw.activated(to(x), "gelu"), O.gelu_erf(z))
    assert ok(lw.activated(to(x), "gelu", row_gate=gd[:, 1]), O.gelu_erf(z) * torch.sigmoid(gate[:, 1:2].double()))
    off = 8
    assert ok(lw.activated(to(x), "gelu_tanh", mul=td[:, off:off + N], mul_rows=rows.int().to(device)), O.gelu_tanh(z) * table[rows, off:off + N].double())
    wide = torch.zeros(M, N + 24, dtype=dtype, device=device)
    lw.activated(to(x), "gelu", out=wide[:, 16:16 + N])
    assert ok(wide[:, 16:16 + N], O.gelu_erf(z)) and (wide[:, :16] == 0).all() and (wide[:, 16 + N:] == 0).all()
    h0 = torch.randn(M, N, generator=g)
    h, copy = h0.clone().to(device), torch.empty(M, N, dtype=dtype, device=device)
    lw.add_to(to(x), h, 1.0, copy=copy)
    assert (h.cpu().double() - h0.double() - z).abs().max() < (2e-5 if dtype == torch.float32 else 1e-4) * (1 + z.abs().max())
    assert ok(copy, h0.double() + z)
    w2 = (r16(N, K) * K ** -0.5).to(torch.bfloat16)
    inter = device == "cuda" and N % 64 == 0
    both = B.interleave_gate_up(to(w), to(w2)) if inter else torch.cat([to(w), to(w2)])
    gu = LinearWeight.from_dense(both, interleaved=inter, act_dtype=dtype)
    gu.exact32 = dtype == torch.float32
    wide.zero_()
    gu.glu(to(x), "gelu_tanh", out=wide[:, 8:8 + N])
    assert ok(wide[:, 8:8 + N], O.gelu_tanh(z) * O.linear(w2.double(), x.double()), 0.05) and (wide[:, :8] == 0).all()


def _case(kind, mx, lens, news, device, dtype, seed=0, strong=(), sinks=None):
    """Cached keys and values of requests with ``lens`` tokens, of which the last ``news`` are this batch's, through ``post`` and
    ``attention``.  ``strong``: (request, query index, key index, length): that query points at that key, in every head."""
    g = torch.Generator().manual_seed(seed)
    H, G, D, V, rot = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], mx.get("rot")
    norms = kind == "attention_2"
    r16 = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    qn, kn = (1.2 + 0.2 * torch.randn(D, generator=g)).to(torch.bfloat16), (1.2 + 0.2 * torch.randn(D, generator=g)).to(torch.bfloat16)
    k, v = [r16(n, G, D) for n in lens], [r16(n, G, V) for n in lens]
    q, gate = [r16(n, H, D) for n in news], torch.randn(sum(news), H, generator=g)
    sinks = torch.randn(H, generator=g) if sinks is None else sinks
    turn = lambda x, w, p: O.rotate(O.rms_norm(x.double(), w.double(), 1e-5), p, rot) if norms else x.double()
    kr = [turn(k[b], kn, torch.arange(n)) for b, n in enumerate(lens)]
    for b, i, j, length in strong:
        at = lens[b] - news[b] + i
        seen = O.rotate(kr[b][j:j + 1], torch.tensor([-at]), rot)[0] if norms else kr[b][j]       # the key seen from the query's position
        for h in range(H):
            d = seen[h // (H // G)] / (qn.double() if norms else 1.0)
            q[b][i, h] = (d * (length / d.norm())).to(torch.bfloat16)
    qr = [turn(q[b], qn, torch.arange(n - m, n)) for b, (n, m) in enumerate(zip(lens, news))]
    want = torch.cat([O.attention_core(qr[b], kr[b], v[b].double(), mx, None if norms else sinks.double()) for b in range(len(lens))])
    if not norms:
        want = want * torch.sigmoid(gate.double())[..., None]
    spec = from_hf_dict(config([((kind, mx), None)])).mixers[0]
    to = lambda t: t.to(device, dtype)
    z = lambda n: torch.zeros(n, 16, dtype=dtype, device=device)
    w, _ = GR.build(spec, z(H * D), z(G * D), z(G * V), None, to(qn) if norms else None, to(kn) if norms else None, None, None if norms else sinks.to(device))
    cos, sin = A.build_rope_tables(rot["dims"], 4096, spec.rope["theta"], None, device) if rot else (None, None)
    # pages are handed out in a shuffled order; they start dirty
    npg = [(n + PAGE - 1) // PAGE for n in lens]
    order = torch.randperm(sum(npg), generator=g).tolist()
    kp = torch.full((sum(npg), PAGE, G, w.dp), 3.0, dtype=dtype, device=device)
    vp = torch.full((sum(npg), PAGE, G, w.vp), -2.0, dtype=dtype, device=device)
    table = torch.zeros((len(lens), max(npg)), dtype=torch.int32)
    for b in range(len(lens)):
        for i in range(npg[b]):
            table[b, i] = order.pop()

    def batch(first, last):
        """Tokens [first[b], last[b]) of every request, and their projection rows."""
        cu, pos, slots, rows = [0], [], [], []
        for b in range(len(lens)):
            n = last[b] - first[b]
            cu.append(cu[-1] + n)
            p = torch.arange(first[b], last[b])
            pos.append(p)
            slots.append(table[b][p // PAGE].long() * PAGE + p % PAGE)
            row = torch.zeros(n, (w.v_col + G * w.vp + 31) // 32 * 32)
            put = lambda c, x, m: row[:, c:c + x.shape[1] * m].view(n, x.shape[1], m)[..., :x.shape[2]].copy_(x.float())
            if first[b] >= lens[b] - news[b]:
                put(0, q[b][first[b] - lens[b] + news[b]:last[b] - lens[b] + news[b]], w.dp)
            put(w.k_col, k[b][first[b]:last[b]], w.dp)
            put(w.v_col, v[b][first[b]:last[b]], w.vp)
            rows.append(row)
        i32 = lambda t: torch.as_tensor(t).to(torch.int32).to(device)
        fb = ForwardBatch(ids=i32(torch.cat(pos)), positions=i32(torch.cat(pos)), slots=i32(torch.cat(slots)), page_table=table.to(device), kv_lens=i32(last),
                          cu_q=i32(cu), cu_q_host=cu, is_decode=all(cu[i + 1] - cu[i] == 1 for i in range(len(lens))), kv_lens_host=list(last))
        return fb, to(torch.cat(rows))

    if any(n > m for n, m in zip(lens, news)):                        # the earlier tokens' keys and values
        fb, proj = batch([0] * len(lens), [n - m for n, m in zip(lens, news)])
        GR.post(w, proj, fb, (kp, vp), cos, sin, 1e-5)
    fb, proj = batch([n - m for n, m in zip(lens, news)], lens)
    GR.post(w, proj, fb, (kp, vp), cos, sin, 1e-5)
    out = torch.full((proj.shape[0], H * w.vp + 16), 7.0, dtype=dtype, device=device)         # a column slice of a wider buffer
    GR.attention(w, proj, (kp, vp), fb, out=out[:, 8:8 + H * w.vp], head_gate=None if norms else gate.to(device))
    assert (out[:, :8] == 7.0).all() and (out[:, 8 + H * w.vp:] == 7.0).all()
    return out[:, 8:8 + H * w.vp].cpu().double().view(-1, H, w.vp)[..., :V], want


def _check(kind, mx, lens, news, where, **kw):
    device, dtype = where
    got, want = _case(kind, mx, lens, news, device, dtype, **kw)
    err = (got - want).abs().amax(-1).amax(-1)
    assert err.max() < (5e-5 if dtype == torch.float32 else 0.1), (err.argmax().item(), err.max().item())


MIXERS = [full(4, 2, 32, 24), full(3, 1, 20, 12, cap=2.0), full(40, 2, 128, 128, cap=30.0), full(2, 2, 256, 256), full(2, 1, 300, 264),
          local(4, 2, 32, 24, 41, 3, 16), local(3, 3, 20, 12, 129, 140, 6), local(40, 2, 128, 128, 1000, 9, 64), local(8, 1, 96, 112, 128, 128, 96),
          local(16, 1, 192, 128, 64, 1, 8), local(2, 2, 64, 200, 77, 200, 64), local(5, 5, 64, 64, 300, 0, 2, cap=0.0), local(2, 1, 300, 264, 90, 20, 20)]


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("kind,mx", MIXERS, ids=lambda m: m if isinstance(m, str) else "-".join(str(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))
                         + "".join(f"-{x}" for x in (m.get("mask") or {}).values()))
def test_attention(kind, mx, where):
    """Decoded tokens, prompt blocks (one and several 128- and 256-row blocks), short portions, and all of them in one batch."""
    _check(kind, mx, [1, 2, 40, 41, 42, 128, 129, 300, 1100], [1] * 9, where)
    _check(kind, mx, [700], [700], where, seed=1)
    _check(kind, mx, [17, 300, 1100, 129, 600], [17, 257, 130, 128, 18], where, seed=2)
    _check(kind, mx, [500, 260, 90, 1030, 33], [1, 200, 2, 300, 16], where, seed=3)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("mx", [local(4, 2, 32, 24, 41, 6, 16, scale=1.0, cap=40.0)[1], local(9, 3, 128, 128, 130, 129, 64, scale=0.5, cap=30.0)[1],
                                local(2, 1, 24, 40, 257, 66, 24, scale=1.0, cap=25.0)[1]], ids=["w41", "w130", "w257"])
def test_far_keys_stand_out(mx, where):
    """One key carries nearly all of a query's weight: the window's first position, the one before it (unseen), the kept tokens' last one
    and the next (unseen), page borders; for decoded rows and for rows of a portion."""
    C, keep = mx["mask"]["size"], mx["mask"]["keep_first"]
    n = 3 * C + 300
    for news in (1, 2, 16, 17, 300) if where[0] == "cuda" else (1, 300):
        for i in sorted({0, news // 2, news - 1}):
            at = n - news + i                                       # position of the query
            for j in {at, at - C + 1, at - C, at - C // 2, 0, keep - 1, keep, keep + 1, (at // PAGE) * PAGE, (at // PAGE) * PAGE - 1, PAGE}:
                if 0 <= j <= at:
                    _check("attention_2", mx, [n, 200], [news, 1], where, seed=j, strong=[(0, i, j, 30.0)])


@pytest.mark.parametrize("where", DEVICES)
def test_far_keys_without_window(where):
    kind, mx = full(4, 2, 32, 24, cap=35.0, scale=1.0)
    for n, news in ((700, 1), (700, 2), (900, 300)):
        for j in (0, 1, 63, 64, PAGE - 1, PAGE, 5 * PAGE - 1, n - news):
            _check(kind, mx, [n, 40], [news, 17], where, seed=j, strong=[(0, 0, j, 6.0), (0, news - 1, j, 6.0)])


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("level", [-30.0, 0.0, 8.0, 30.0])
def test_sinks_show(level, where):
    """Sinks that take nothing, some and nearly all of the weight; below and above every score, for one key and for many."""
    kind, mx = full(6, 2, 32, 24, cap=12.0)
    sinks = level + torch.tensor([0.0, 1.0, -1.0, 2.0, -2.0, 0.5])
    for lens, news in (([1, 2, 200, 520], [1, 1, 1, 1]), ([1, 200, 520], [1, 200, 300])):
        device, dtype = where
        got, want = _case(kind, mx, lens, news, device, dtype, sinks=sinks)
        floor = want.abs().amax()
        assert (got - want).abs().max() < (5e-5 if dtype == torch.float32 else 0.02) * floor + 1e-9
        if level == 30.0:
            assert floor < 1e-4                                     # (what is left is compared relative to itself)


@pytest.mark.parametrize("where", DEVICES)
def test_soft_cap_shows(where):
    """Scores far beyond the cap on either side: many keys end up alike."""
    for kind, mx in (full(4, 2, 32, 24, cap=1.5, scale=1.0), local(4, 2, 32, 24, 60, 4, 8, cap=1.5, scale=1.0)):
        _check(kind, mx, [300, 70], [300, 1], where)


@pytest.mark.parametrize("where", DEVICES)
def test_many_decoded_rows(where):
    """More rows than one call of the decode kernel takes."""
    n = 40 if where[0] == "cuda" else 3
    _check(*local(2, 1, 32, 32, 50, 5, 16), [200 + b for b in range(n)], [16] * n, where)
    _check(*full(2, 1, 32, 32), [200 + b for b in range(n)], [16] * n, where)


def _cell_case(mx, parts, device, dtype, seed=0, i_shift=-0.5, f_shift=3.0, z_scale=2.0, eps=0.01):
    """Requests cut into ``parts`` (lists of portion lengths, one step each), in state slots handed out in reverse; a step is one batch.
    ``eps`` is not small, so that the size of the outputs shows behind their norm."""
    g = torch.Generator().manual_seed(seed)
    H, D, V, cap = mx["heads"], mx["dim"], mx["vdim"], mx["gate_cap"]
    r16 = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    nw, bias = (1 + 0.2 * r16(H * V)).to(torch.bfloat16), torch.cat([r16(H) + i_shift, r16(H) + f_shift]).to(torch.bfloat16)
    lens = [sum(p) for p in parts]
    x = [dict(q=r16(n, H * D), k=r16(n, H * D), v=r16(n, H * V), g=r16(n, H * V)) for n in lens]
    z = [z_scale * torch.randn(n, 2 * H, generator=g) for n in lens]
    want = []
    for t, zz in zip(x, z):
        n = t["q"].shape[0]
        rs = lambda m, d: m.double().reshape(n, H, d)
        soft = cap * torch.tanh((zz.double() + bias.double()) / cap)
        o, _ = O.mlstm_recurrence(rs(t["q"], D) * D ** -0.5, rs(t["k"], D), rs(t["v"], V), soft[:, :H], torch.nn.functional.logsigmoid(soft[:, H:]))
        want.append(O.unit_rms(o, eps).reshape(n, H * V) * nw.double() * torch.sigmoid(t["g"].double()))
    to = lambda t: t.to(device, dtype)
    zero = lambda n: torch.zeros(n, 16, dtype=dtype, device=device)
    w, _ = ML.build(MLSTMSpec(H, D, V, cap), zero(H * D), zero(H * D), zero(H * V), zero(H * V), to(bias[:H]), to(bias[H:]), to(nw))
    state = torch.zeros((len(parts) + 1, H, ML.state_len(D, V)), device=device)
    state[-1] = 5.0                                                   # a slot nobody uses
    done, got = [0] * len(parts), [[] for _ in parts]
    for s in range(max(len(p) for p in parts)):
        reqs = [b for b in range(len(parts)) if s < len(parts[b]) and parts[b][s]]
        cu, rows, gates = [0], [], []
        for b in reqs:
            n = parts[b][s]
            cu.append(cu[-1] + n)
            row = torch.zeros(n, (w.cols[-1] + H * V + 7 + 31) // 32 * 32)
            for key, c in zip("qkvg", w.cols):
                m = x[b][key][done[b]:done[b] + n]
                row[:, c:c + m.shape[1]] = m.float()
            rows.append(row)
            gates.append(z[b][done[b]:done[b] + n])
            done[b] += n
        slots = [len(parts) - 1 - b for b in reqs]
        i32 = lambda t: torch.tensor(t, dtype=torch.int32, device=device)
        fb = ForwardBatch(ids=None, positions=None, slots=None, page_table=i32([[0]]), kv_lens=None, cu_q=i32(cu), cu_q_host=cu, is_decode=cu == list(range(len(cu))),
                          state_slots=i32(slots), state_slots_host=slots)
        y = ML.mix(w, to(torch.cat(rows)), torch.nn.functional.pad(torch.cat(gates), (0, 5)).to(device)[:, :2 * H], fb, state, eps).cpu().double()
        for i, b in enumerate(reqs):
            got[b].append(y[cu[i]:cu[i + 1]])
    assert (state[-1] == 5.0).all()
    return torch.cat([torch.cat(t) for t in got]), torch.cat(want)


def _check_cell(mx, parts, where, over=0.0, **kw):
    """``over``: the fraction of rows that may miss the limit (a denominator that nearly cancels)."""
    device, dtype = where
    got, want = _cell_case(mx, parts, device, dtype, **kw)
    assert torch.isfinite(got).all()
    err = (got - want).abs().amax(-1) / (1 + want.abs().amax(-1))
    limit = 1e-4 if dtype == torch.float32 else 0.03
    assert (err >= limit).double().mean() <= over and err.max() < (100 if over else 1) * limit, (err.argmax().item(), err.max().item())


CELLS = [cell(3, 24, 40)[1], cell(1, 8, 8, 1.0)[1], cell(2, 20, 12, 30.0)[1], cell(4, 128, 128, 15.0)[1], cell(2, 64, 192)[1], cell(1, 256, 64)[1], cell(2, 192, 128)[1],
         cell(2, 40, 256)[1], cell(1, 256, 256)[1], cell(1, 300, 20)[1]]


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("mx", CELLS, ids=lambda v: "-".join(str(x) for x in v.values()))
def test_matrix_memory(mx, where):
    """Whole prompts, portions of every kind (chunk borders just missed), single tokens, and batches of them."""
    n = 1 if where[0] == "cpu" else 3
    _check_cell(mx, [[129 * n]], where)
    _check_cell(mx, [[1] * 12, [1] * 12, [1] * 9], where, seed=1)
    _check_cell(mx, [[127, 1, 2, 128, 1], [2, 2, 70, 1, 1], [1, 1, 1, 1, 1], [64, 65, 0, 3, 17], [128 * n, 1, 15, 33, 2]], where, seed=2)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("kw", [dict(f_shift=-40.0), dict(f_shift=60.0), dict(i_shift=40.0), dict(i_shift=-40.0, f_shift=60.0), dict(z_scale=30.0)], ids=str)
def test_gate_extremes(kw, where):
    """Heads that forget within a token and heads that never do, input gates at their caps: the running maximum grows, falls and stands
    still, either side of the denominator is taken, and nothing overflows."""
    for cap in (2.0, 14.0):
        _check_cell(cell(2, 32, 24, cap)[1], [[200, 1, 1, 40], [7, 128, 1, 1]], where, over=0.01, **kw)


@pytest.mark.parametrize("where", DEVICES)
def test_first_token_survives(where):
    """With forget gates of almost one and a strong first input gate, the first token's value is still read after many chunks."""
    for parts in ([[500]], [[2, 250, 200, 48]], [[128] * 3 + [1] * 44]):
        _check_cell(cell(1, 16, 8, 12.0)[1], parts, where, f_shift=30.0, z_scale=0.5, seed=4)


def test_the_two_sides_of_the_denominator():
    """The oracle itself: a lone token is read back through max(|n . q|, e^-m), with m that starts at zero."""
    q, k, v = torch.ones(1, 1, 1).double(), torch.full((1, 1, 1), 0.5).double(), torch.full((1, 1, 1), 3.0).double()
    for i in (-4.0, 0.0, 2.0):
        o, (S_, n, m) = O.mlstm_recurrence(q, k, v, torch.full((1, 1), i).double(), torch.full((1, 1), -1.0).double())
        m_want = max(-1.0, i)
        a = 2.718281828459045 ** (i - m_want)
        assert abs(o.item() - a * 1.5 / (max(a * 0.5, 2.718281828459045 ** -m_want) + 1e-6)) < 1e-9 and m.item() == m_want


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("experts,top,groups", [(6, 2, (3, 1)), (40, 5, (8, 3)), (64, 6, (4, 4)), (9, 3, (9, 3)), (12, 1, (1, 1)), (16, 4, (2, 1)), (512, 8, (32, 5)), (600, 3, (3, 2))])
def test_grouped_choice(experts, top, groups, where):
    """Best scores of the groups whose largest score is best, as columns of a wider matrix of logits; weights are softmax scores of all."""
    device = where[0]
    g = torch.Generator().manual_seed(experts)
    z = torch.randn(50, experts + 7, generator=g) * 3
    idx, wts = MOE.route_topk(z.to(device)[:, 4:4 + experts], None, top, 0, False, groups[0], groups[1], group_max=True)
    s = torch.softmax(z[:, 4:4 + experts].double(), dim=-1)
    router = {"top": top, "groups": {"count": groups[0], "keep": groups[1]}}
    for t in range(50):
        want = O.choose(s[t], router)
        assert sorted(idx[t].tolist()) == sorted(want)
        assert (s[t][idx[t].long().cpu()] - wts[t].cpu().double()).abs().max() < 1e-6


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("shape", [(6, 3, 48, 160, 72, None), (9, 1, 112, 256, None, (3, 2)), (64, 6, 64, 384, 128, (8, 4)), (1, 1, 8, 72, 8, None), (8, 8, 200, 64, 33, (2, 2))], ids=str)
@pytest.mark.parametrize("rows", [1, 7, 300, 900])
def test_parallel_block_with_experts(tmp_path, shape, rows, where):
    """One layer: router, plan, experts without gate branch, gated shared expert, mixer, their joint product and combine, residual."""
    device, dtype = where
    E, top, ff, width, shared, groups = shape
    rows = rows if where[0] == "cuda" else min(rows, 7)
    cfg = config([(cell(1, 8, 8), moe(E, top, ff, shared, groups))], width=width, vocab=112)
    w = O.random_weights(cfg, seed=E)
    m = load_model(save(tmp_path / "m", cfg, w), device=device, dtype=dtype)
    g = torch.Generator().manual_seed(rows)
    x = torch.randn(rows, width, generator=g).to(torch.bfloat16)
    wd = {k: v.double() for k, v in w.items()}
    xd = x.double()
    s = xd @ wd["l0.mlp.router"].T
    clear = torch.ones(rows, dtype=torch.bool)
    per = E // (groups[0] if groups else 1)
    for t in range(rows):
        best = s[t].view(-1, per).amax(-1).sort(descending=True).values
        keep = groups[1] if groups else 1
        kept = torch.cat([s[t].view(-1, per)[i] for i in s[t].view(-1, per).amax(-1).argsort(descending=True)[:keep]]).sort(descending=True).values
        clear[t] = (keep >= best.numel() or best[keep - 1] - best[keep] > 1e-4) and (top >= kept.numel() or kept[top - 1] - kept[top] > 1e-4)
    i32 = lambda t: torch.tensor(t, dtype=torch.int32, device=device)
    fb = ForwardBatch(ids=i32([3] * rows), positions=i32(list(range(rows))), slots=i32([-1] * rows), page_table=i32([[0]]), kv_lens=i32([rows]), cu_q=i32([0, rows]),
                      cu_q_host=[0, rows], kv_lens_host=[rows], state_slots=i32([0]), state_slots_host=[0])
    state = torch.zeros((1, 1, ML.state_len(8, 8)), device=device)
    h = xd.float().to(device)
    h, y = m._parallel_layer(m.layers[0], x.to(device, dtype), fb, (None, state), h, 0)
    want = xd + O.mlstm(xd, wd, "l0.mix.", cfg["layers"][0]["mixer"], 1e-5) + O.moe(xd, wd, "l0.mlp.", cfg["layers"][0]["mlp"])
    tol = 5e-5 if dtype == torch.float32 else 0.03
    assert clear.double().mean() > 0.9
    assert (h.cpu().double() - want)[clear].abs().max() < tol * (1 + want.abs().max())
    ref = O.rms_norm(want, wd["final.norm"], 1e-5)
    assert (y.cpu().double() - ref)[clear].abs().max() < tol * (1 + ref.abs().max())


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("what", ["loop", "step", "side", "kept", "sink", "cap", "gate"])
def test_every_part_counts(models, what, where):
    """The reference with one part taken out is far from the framework (so the other tests see it)."""
    device, dtype = where
    cfg, w, path = models("mixed")
    toks = prompt("mixed", 190, 60)
    rp = Replay(open_engine(path, dtype, 256, device))
    got = rp.step([("a", toks, list(range(190)))], ["a"]).double()
    cut, cw = json.loads(json.dumps(cfg)), dict(w)
    if what == "loop":
        cut["loop"]["times"] = 2
    elif what == "step":
        cw["loop.step"] = w["loop.step"] * 0
    elif what == "side":
        cw["side.embed"] = w["side.embed"].roll(24, dims=1)              # another layer's part
    elif what == "kept":
        cut["layers"][0]["mixer"]["mask"]["keep_first"] = 0
    elif what == "sink":
        cw["l2.mix.sink"] = w["l2.mix.sink"] - 50
    elif what == "cap":
        cut["layers"][2]["mixer"]["softcap"] = 0.7
    else:
        cw["l2.mix.g"] = w["l2.mix.g"] * 0
    far, near = O.forward(cut, cw, toks), oracle("mixed", toks)
    worst = lambda a: ((got - a).pow(2).mean(-1).sqrt() / near.pow(2).mean(-1).sqrt()).max().item()
    assert worst(near) < (3e-5 if dtype == torch.float32 else 0.05) and worst(far) > 0.03 and worst(far) > 2 * worst(near), (worst(near), worst(far))


# ---------------------------------------------------------------------------------------------------
# configuration, scheduler, sampling
# ---------------------------------------------------------------------------------------------------
def test_layers_and_their_pools(models):
    cfg, w, path = models("mixed")
    eng = open_engine(path, torch.float32, 256, "cpu")
    m, pools = eng.model, eng.runner.kv.pools
    assert m.cfg.layer_runs == [0, 1, 2, 1, 2, 1, 2, 3, 4] and m.cfg.pass_starts == [None, 0, None, 1, None, 2, None, None, None]
    assert [type(x) for x in m.cfg.mixers] == [AttnSpec, MLSTMSpec, AttnSpec] + [MLSTMSpec, AttnSpec] * 2 + [MLSTMSpec, AttnSpec]
    assert m.layers[3] is m.layers[1] and pools[3][1] is not pools[1][1] and pools[4][0] is not pools[2][0]        # one set of weights, a cache per pass
    assert pools[0][0].shape[2:] == (3, 40) and pools[0][1].shape[2:] == (3, 24) and pools[8][1].shape[2:] == (4, 72)
    assert pools[1][1].shape == (5, 3, ML.state_len(24, 40)) and pools[1][1].dtype == torch.float32
    assert m.kv_bytes_per_page() == 4 * PAGE * (3 * 64 + 3 * 2 * 64 + 4 * 136)
    assert m.linear_state_bytes_per_slot() == 4 * (9 * ML.state_len(24, 40) + 2 * ML.state_len(64, 16))


def test_unknown_parts_are_refused():
    for change in (lambda c: c["layers"][0].update(type="something_else"), lambda c: c["layers"][1]["mlp"].update(kind="other"), lambda c: c["loop"].update(stop=9),
                   lambda c: c["loop"].update(times=0)):
        cfg = json.loads(json.dumps(CONFIGS["ones"]))
        change(cfg)
        with pytest.raises((NotImplementedError, ValueError)):
            from_hf_dict(cfg)


@pytest.mark.parametrize("where", DEVICES)
def test_greedy_generation(models, where):
    """The engine's own scheduler: chunked prompts beside decoding requests, arg-max of the plain model; the same prompts again through
    used pages and state slots."""
    device, dtype = where
    name, n_new = "mixed", 6
    cfg, w, path = models(name)
    m = load_model(path, device=device, dtype=dtype)
    eng = LLMEngine(m, EngineConfig(max_batch=2, max_context=512, chunked_prefill_size=50), num_pages=20)
    prompts = [prompt(name, k, 20) for k in (1, 60, 133)]
    outs = eng.generate(prompts, GenerationConfig(max_new_tokens=n_new, ignore_eos=True))
    for p, out in zip(prompts, outs):
        assert len(out) == n_new
        logits = O.forward(cfg, w, p + out[:-1])[len(p) - 1:]
        for k, t in enumerate(out):                                 # a near tie may fall either way in 16 bits
            gap = (logits[k].max() - logits[k][t]).item()
            assert gap < (1e-4 if dtype == torch.float32 else 0.1), (k, gap)
    again = eng.generate(prompts, GenerationConfig(max_new_tokens=n_new, ignore_eos=True))
    assert again == outs or dtype != torch.float32


def test_speculative_generation_matches_greedy(models):
    """Drafts by prompt lookup: rejected drafts leave the recurrent state as if they had never been read."""
    m = load_model(models("bare")[2], device="cpu", dtype=torch.float32)
    prompts, outs = [prompt("bare", 9, 5) * 4, [7, 8, 9] * 10], []
    for spec in ("", "ngram"):
        eng = LLMEngine(m, EngineConfig(max_batch=2, max_context=256, speculative=spec), num_pages=8)
        outs.append(eng.generate(prompts, GenerationConfig(max_new_tokens=12, ignore_eos=True)))
    assert outs[0] == outs[1]


def test_layers_without_pages(tmp_path):
    """A stack of recurrent layers only: no page pools, the scheduler runs on state slots."""
    cfg = config([(cell(2, 16, 16), moe(2, 1, 16)), (cell(1, 24, 8), None)], width=64, vocab=64, loop=(1, 2, 2))
    w = O.random_weights(cfg, seed=1)
    m = load_model(save(tmp_path / "m", cfg, w), device="cpu", dtype=torch.float32)
    eng = LLMEngine(m, EngineConfig(max_batch=2, max_context=256, max_tokens=512))
    toks = list(range(20))
    out = eng.generate([toks, toks[:3]], GenerationConfig(max_new_tokens=3, ignore_eos=True))
    logits = O.forward(cfg, w, toks + out[0][:-1])[19:]
    assert [x.argmax().item() for x in logits] == out[0]


@gpu
@pytest.mark.parametrize("wdtype", ["int8", "fp8"])
def test_quantised_weights(models, wdtype):
    """Run-time weight formats: the same model with coarser weights."""
    cfg, w, path = models("wide")
    m = load_model(path, device="cuda", wdtype=wdtype)
    rp = Replay(LLMEngine(m, EngineConfig(max_batch=4, max_context=256, prefix_cache=False), num_pages=4))
    toks = prompt("wide", 150, 40)
    got = torch.cat([rp.step([("a", toks[:140], list(range(140)))])] + [rp.step([("a", toks[i:i + 1], [0])]) for i in range(140, 150)])
    assert_close(got, oracle("wide", toks), torch.bfloat16, 0.25, over=0.1)


def test_public_entry_points(models):
    from fastllm_b200 import llm
    from fastllm_b200.models import preset, random_init

    cfg, w, path = models("mixed")
    toks = prompt("mixed", 12, 50)
    old = llm._resolve_device()
    llm.set_device_map("cpu")
    try:
        m = llm.model(str(path))
        out = list(m.stream_response_raw(toks, max_length=4, do_sample=False))
        m.release_memory()
    finally:
        llm.set_device_map(str(old))
    want = O.forward(cfg, w, (toks + out)[:-1])[len(toks) - 1:]
    assert len(out) == 4 and all((want[k].max() - want[k][t]) < 0.1 for k, t in enumerate(out))
    tiny = random_init(preset("tiny-vuripel"), "cpu", torch.float32)
    outs = LLMEngine(tiny, EngineConfig(max_batch=2, max_context=256), num_pages=8).generate([[1, 2, 3]], GenerationConfig(max_new_tokens=3, ignore_eos=True))
    assert len(outs[0]) == 3


def test_command_line_replay(models, tmp_path, capsys, monkeypatch):
    import io
    import sys

    from fastllm_b200.engine import replay as R

    cfg, w, path = models("ones")
    toks = prompt("ones", 9, 30)
    lines = [{"step": 0, "entries": [{"id": "x", "tokens": toks[:5], "want": [1, 4]}], "end": []},
             {"step": 1, "entries": [{"id": "x", "tokens": toks[5:8], "want": []}], "end": []},
             {"step": 2, "entries": [{"id": "x", "tokens": toks[8:], "want": [0]}], "end": ["x"]}]
    monkeypatch.setattr(sys, "stdin", io.StringIO("\n".join(json.dumps(s) for s in lines) + "\n"))
    assert R.main(["--model", str(path), "--dtype", "float32", "--out", str(tmp_path), "--max-tokens", "64", "--device", "cpu"]) == 0
    assert [s for s in capsys.readouterr().out.splitlines() if s.startswith("done")] == ["done 0", "done 1", "done 2"]
    want = O.forward(cfg, w, toks)
    read = lambda i: torch.frombuffer(bytearray((tmp_path / f"{i}.f32").read_bytes()), dtype=torch.float32).view(-1, cfg["vocab"])
    assert_close(read(0), want[[1, 4]], torch.float32)
    assert not (tmp_path / "1.f32").exists()
    assert_close(read(2), want[8:], torch.float32)
