"""Vilulorn (gated linear attention, chunked grouped-query attention with shared keys and values, sigmoid-scored experts on scaled
inputs, normalised sub-layer outputs, learned positions) against its plain statement.

Every case builds a small random model of its own.  The CPU runs use the framework's PyTorch operator definitions (scheduling,
cache, loading and the model itself); the GPU runs the kernels, in float32 and bfloat16.
"""
import json

import pytest
import torch

from . import listed_common as LC
from . import vilulorn_oracle as O
from .listed_common import DEVICES, PAGE, assert_close, few_threads, portions, save  # noqa: F401
from fastllm_b200.engine import EngineConfig, GenerationConfig, LLMEngine
from fastllm_b200.engine.replay import Replay, open_engine
from fastllm_b200.loader.hf import load_model
from fastllm_b200.models.config import AttnSpec, GLASpec, from_hf_dict
from fastllm_b200.models.decoder import ForwardBatch
from fastllm_b200.ops import attention as A
from fastllm_b200.ops import gla as GLA
from fastllm_b200.ops import grouped as GR
from fastllm_b200.ops import moe as MOE
from fastllm_b200.ops import stream32 as S

gpu = pytest.mark.gpu


def attn(heads, kv, dim, vdim, chunk, rot, scale=None, src=None, base=1e4, scaling=None):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or 0.7 * dim ** -0.5, "mask": {"size": chunk},
         "rot": {"base": base, "dims": rot, "scaling": scaling or {"factor": 3.0, "low": 1.5, "high": 5.0, "original": 96}}}
    if src is not None:
        m["kv_from"] = src
    return "attention", m


def gla(heads, dim, vdim, tau):
    return "gla", {"heads": heads, "dim": dim, "vdim": vdim, "tau": tau}


def moe(experts, top, ff, limit):
    return {"kind": "moe", "expert": {"ff": ff, "limit": limit}, "router": {"experts": experts, "top": top}}


def config(layers, width=160, vocab=304, eps=1e-5, positions=640):
    return {"architecture": "Vilulorn", "vocab": vocab, "width": width, "norm": {"eps": eps}, "max_positions": positions,
            "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}


CONFIGS = {
    # every expert is taken (no close calls in 16 bits); two chunk sizes over one cache, a layer without feed-forward
    "mixed": config([(attn(6, 3, 40, 24, 50, 16), moe(3, 3, 48, 1.5)), (gla(3, 24, 40, 8.0), None), (attn(6, 3, 40, 24, 77, 16, src=0), moe(2, 2, 112, 0.8)),
                     (gla(2, 64, 16, 16.0), moe(3, 3, 64, 4.0)), (attn(4, 4, 64, 72, 150, 64), None)]),
    # nothing is a multiple of anything the kernels tile; the first layer is recurrent and the donor comes later
    "odd": config([(gla(3, 20, 12, 5.0), moe(3, 3, 75, 1.1)), (attn(3, 1, 20, 12, 19, 6, scale=0.3), None), (attn(3, 1, 20, 12, 37, 6, scale=0.2, src=1), moe(2, 2, 30, 2.0)),
                   (gla(1, 33, 50, 1.0), None)], width=148, vocab=331, eps=1e-4),
    # heads of a served size: sixteen query heads per key head, whole tensor-core tiles, wide states
    "wide": config([(attn(32, 2, 128, 128, 200, 64), moe(2, 2, 128, 3.0)), (gla(4, 128, 128, 16.0), moe(4, 4, 64, 2.5)), (attn(32, 2, 128, 128, 333, 64, src=0), None),
                    (gla(2, 256, 192, 12.0), None), (attn(24, 1, 192, 256, 130, 192), None)], width=256, vocab=512),
    # one head, one expert, chunks of one token, a decay power of one
    "ones": config([(gla(1, 8, 8, 1.0), moe(1, 1, 8, 1.0)), (attn(1, 1, 8, 8, 1, 8), moe(1, 1, 8, 1.0))], width=64, vocab=64),
    # experts are chosen, more of them than a tile of router columns
    "routed": config([(attn(4, 2, 32, 32, 64, 16), moe(40, 3, 64, 2.0)), (gla(2, 32, 32, 16.0), moe(7, 1, 40, 1.0))], width=128, vocab=256),
}
RANKS = {"odd": 5, "wide": 40, "ones": 1}
OVER = {"routed": 0.5}
_CACHE: dict = {}


def weights(name):
    if name not in _CACHE:
        _CACHE[name] = O.random_weights(CONFIGS[name], seed=len(name), rank=RANKS.get(name, 16))
    return _CACHE[name]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, weights, checkpoint folder); the folders are written once."""
    root, out = tmp_path_factory.mktemp("vilulorn"), {}

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
    reqs = {str(n): prompt(name, n) for n in (1, 2, 17, 130, 300)}
    replay(models, name, where, reqs, [[(r, len(t))] for r, t in reqs.items()], 384)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_token_by_token(models, name, where):
    """From the first token on, across page borders and past every chunk that is shorter."""
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
# chunk edges: with one attention layer, a token reaches exactly the rows of its own chunk behind it
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("chunk", [1, 2, 31, 64, 100, 128, 129])
def test_chunk_edge(tmp_path, chunk, where):
    device, dtype = where
    cfg = config([(attn(2, 1, 32, 32, chunk, 16), None)], width=64, vocab=96)
    w = O.random_weights(cfg, seed=chunk)
    path = save(tmp_path / "m", cfg, w)
    k = (PAGE if chunk < PAGE else chunk) // chunk + 1                # the second chunk that ends behind the first page's border
    p, end, n = k * chunk, (k + 1) * chunk, (k + 1) * chunk + 40      # first position of that chunk, of the next one
    g = torch.Generator().manual_seed(chunk)
    base = torch.randint(0, 96, (n,), generator=g).tolist()
    w64 = {kk: v.double() for kk, v in w.items()}
    ref = O.forward(cfg, w64, base)
    # the substitute is the token that moves the chunk's last row most
    best = max(range(96), key=lambda t: (O.forward(cfg, w64, base[:p] + [t] + base[p + 1:end])[-1] - ref[end - 1]).abs().max().item())
    other = base[:p] + [best] + base[p + 1:]
    want = (O.forward(cfg, w64, other) - ref).abs().amax(-1)
    assert want[:p].max() == 0 and want[end:].max() == 0 and want[end - 1] > 0
    eng = open_engine(path, dtype, 512, device)
    for cut in ([n], [p + chunk // 2 + 1, n - p - chunk // 2 - 1], [max(1, p - 1)] + [1] * (n - max(1, p - 1)) if device == "cuda" or chunk < 40 else [n]):
        outs = []
        for seq in (base, other):
            rp, at, rows = Replay(eng), 0, []
            for c in cut:
                rows.append(rp.step([("r", seq[at:at + c], list(range(c)))], ["r"] if at + c == n else []))
                at += c
            outs.append(torch.cat(rows))
        diff = (outs[0] - outs[1]).abs().amax(-1)
        noise = 1e-5 if dtype == torch.float32 else 1e-6                # rows that do not see the token are computed alike, bit for bit
        assert diff[:p].max() <= noise and diff[end:].max() <= noise, "a row outside the chunk sees the token"
        assert (diff[end - 1] - want[end - 1]).abs() < 0.05 * want[end - 1] + (1e-4 if dtype == torch.float32 else 0.05), "the chunk's last row misses the token"


# ---------------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("width", [64, 148, 75])
def test_embedding_and_learned_positions(width, where):
    device, dtype = where
    g = torch.Generator().manual_seed(width)
    table, pt, nw = (torch.randn(*s, generator=g).to(torch.bfloat16) for s in ((50, width), (40, width), (width,)))
    ids, pos = torch.randint(0, 50, (6,), generator=g), torch.tensor([0, 1, 17, 38, 39, 39])
    to = lambda t: t.to(device, dtype)
    want = table[ids].double() + pt[pos].double()
    tol = 2e-6 if dtype == torch.float32 else 0.03
    for norm in (None, nw):
        h, y = S.embed_pos_norm(ids.int().to(device), pos.int().to(device), to(table), None, to(norm) if norm is not None else None, 1e-5, pos_table=to(pt))
        assert (h.cpu().double() - want).abs().max() < 2e-6 and y.dtype == dtype
        ref = want if norm is None else O.rms_norm(want, nw.double(), 1e-5)
        assert (y.cpu().double() - ref).abs().max() < tol * ref.abs().max()


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("width", [8, 76, 201, 512])
@pytest.mark.parametrize("post,nxt", [(1, 0), (1, 1), (0, 0), (0, 1)])
def test_output_norm_and_residual(width, post, nxt, where):
    """Plain outputs and expert combines (a pair that is not held, weights, shared rows) onto the residual, with and without the norms."""
    device, dtype = where
    g = torch.Generator().manual_seed(width)
    r = lambda *s: torch.randn(*s, generator=g)
    h0, y, ys, sh = r(9, width), r(9, width).to(torch.bfloat16), r(20, width).to(torch.bfloat16), r(9, width).to(torch.bfloat16)
    pw, nw = ((1 + 0.3 * r(width)).to(torch.bfloat16) for _ in range(2))
    pos = torch.randint(0, 20, (9, 3), generator=g, dtype=torch.int32)
    pos[2, 1] = -1
    wts = torch.rand(9, 3, generator=g)
    to = lambda t: t.to(device, dtype)
    tol = 3e-5 if dtype == torch.float32 else 0.03

    def check(out, h, z):
        z = O.rms_norm(z, pw.double(), 1e-4) if post else z
        want = h0.double() + 0.7 * z
        assert (h.cpu().double() - want).abs().max() < 2e-5 * (1 + want.abs().max())
        ref = O.rms_norm(want, nw.double(), 1e-4) if nxt else want
        assert out.dtype == dtype and (out.cpu().double() - ref).abs().max() < tol * (1 + ref.abs().max())

    h = h0.clone().to(device)
    check(S.add_norm(h, to(y), to(pw) if post else None, to(nw) if nxt else None, 1e-4, 0.7), h, y.double())
    h = h0.clone().to(device)
    out = S.moe_combine_norm(to(ys), pos.to(device), wts.to(device), 1.0, to(sh), h, to(nw) if nxt else None, 0.7, 1e-4, post_w=to(pw) if post else None, dtype=dtype)
    z = torch.where(pos[..., None] >= 0, ys.double()[pos.clamp(min=0).long()] * wts.double()[..., None], torch.zeros(())).sum(1) + sh.double()
    check(out, h, z)


@pytest.mark.parametrize("where", DEVICES)
def test_rotary_frequencies(where):
    """Kept, blended and slowed-down wavelengths, and the degenerate forms of the scaling."""
    for dims, base, sc in ((32, 1e4, {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 128}), (64, 5e5, {"factor": 2.5, "low": 2.0, "high": 3.0, "original": 1000}),
                           (8, 100.0, {"factor": 1.0, "low": 1.0, "high": 1.0, "original": 30}), (16, 1e4, None)):
        _, m = attn(1, 1, dims, 8, 4, dims, base=base)
        m["rot"]["scaling"] = sc
        spec = from_hf_dict(config([(("attention", m), None)])).mixers[0]
        cos, sin = A.build_rope_tables(dims, 300, spec.rope["theta"], spec.rope["scaling"], where[0])
        ang = torch.arange(300, dtype=torch.float64)[:, None] * torch.tensor(O.rotary_frequencies(m["rot"]), dtype=torch.float64)
        assert (cos.cpu().double() - ang.cos()).abs().max() < 1e-6 and (sin.cpu().double() - ang.sin()).abs().max() < 1e-6
    plain = O.rotary_frequencies({"base": 1e4, "dims": 32})
    slow = O.rotary_frequencies({"base": 1e4, "dims": 32, "scaling": {"factor": 8.0, "low": 1.0, "high": 4.0, "original": 128}})
    assert slow[0] == plain[0] and slow[-1] == plain[-1] / 8 and any(p / 8 < s < p for p, s in zip(plain, slow))


def _case(mx, lens, news, device, dtype, seed=0, strong=()):
    """Cached keys and values of requests with ``lens`` tokens, of which the last ``news`` are this batch's, through ``post`` and
    ``attention``.  ``strong``: (request, query index, key index, score): that query meets that key with this score in every head."""
    g = torch.Generator().manual_seed(seed)
    H, G, D, V, dims = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], mx["rot"]["dims"]
    r16 = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    qn, kn = (1.2 + 0.2 * torch.randn(D, generator=g)).to(torch.bfloat16), (1.2 + 0.2 * torch.randn(D, generator=g)).to(torch.bfloat16)
    k, v = [r16(n, G, D) for n in lens], [r16(n, G, V) for n in lens]
    q, gate = [r16(n, H, D) for n in news], [r16(n, H * V) for n in news]
    turn = lambda x, w, p: O.rotate(O.rms_norm(x.double(), w.double(), 1e-5), p, mx["rot"])
    kr = [turn(k[b], kn, torch.arange(n)) for b, n in enumerate(lens)]
    if strong:
        # norms fix the length of a query, so the key is what stands out: queries that point at it, and its norm weight made large
        for b, i, j, boost in strong:
            at = lens[b] - news[b] + i
            inv = O.rotate(kr[b][j:j + 1], torch.tensor([-at]), mx["rot"])[0]       # the key seen from the query's position
            for h in range(H):
                d = inv[h // (H // G)] / qn.double()
                q[b][i, h] = (d * (boost / d.norm())).to(torch.bfloat16)
    qr = [turn(q[b], qn, torch.arange(n - m, n)) for b, (n, m) in enumerate(zip(lens, news))]
    want = torch.cat([O.chunked_core(qr[b], kr[b], v[b].double(), gate[b].double(), mx) for b in range(len(lens))])
    spec = from_hf_dict(config([(("attention", mx), None)])).mixers[0]
    to = lambda t: t.to(device, dtype)
    z = lambda n: torch.zeros(n, 16, dtype=dtype, device=device)
    w, _ = GR.build(spec, z(H * D), z(G * D), z(G * V), z(H * V), to(qn), to(kn))
    cos, sin = A.build_rope_tables(dims, 4096, spec.rope["theta"], spec.rope["scaling"], device) if dims else (None, None)
    # pages are handed out in a shuffled order; they start dirty
    npg = [(n + PAGE - 1) // PAGE for n in lens]
    order = torch.randperm(sum(npg), generator=g).tolist()
    kp = torch.full((sum(npg), PAGE, G, w.dp), 3.0, dtype=dtype, device=device)
    vp = torch.full((sum(npg), PAGE, G, w.vp), -2.0, dtype=dtype, device=device)
    table = torch.zeros((len(lens), max(npg)), dtype=torch.int32)
    for b in range(len(lens)):
        for i in range(npg[b]):
            table[b, i] = order.pop()
    mv = lambda t: t.to(device)

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
            new = slice(first[b] - lens[b] + news[b], last[b] - lens[b] + news[b]) if first[b] >= lens[b] - news[b] else None
            if new is not None:
                put(0, q[b][new], w.dp)
                put(w.gate_col, gate[b][new].view(n, H, V), w.vp)
            put(w.k_col, k[b][first[b]:last[b]], w.dp)
            put(w.v_col, v[b][first[b]:last[b]], w.vp)
            rows.append(row)
        i32 = lambda t: mv(torch.as_tensor(t).to(torch.int32))
        fb = ForwardBatch(ids=i32(torch.cat(pos)), positions=i32(torch.cat(pos)), slots=i32(torch.cat(slots)), page_table=mv(table), kv_lens=i32(last), cu_q=i32(cu),
                          cu_q_host=cu, is_decode=all(cu[i + 1] - cu[i] == 1 for i in range(len(lens))), kv_lens_host=list(last))
        return fb, to(torch.cat(rows))

    if any(n > m for n, m in zip(lens, news)):                        # the earlier tokens' keys and values
        fb, proj = batch([0] * len(lens), [n - m for n, m in zip(lens, news)])
        GR.post(w, proj, fb, (kp, vp), cos, sin, 1e-5)
    fb, proj = batch([n - m for n, m in zip(lens, news)], lens)
    GR.post(w, proj, fb, (kp, vp), cos, sin, 1e-5)
    got = GR.attention(w, proj, (kp, vp), fb).cpu().double().view(-1, H, w.vp)[..., :V].reshape(-1, H * V)
    return got, want


def _check(mx, lens, news, where, **kw):
    device, dtype = where
    got, want = _case(mx, lens, news, device, dtype, **kw)
    err = (got - want).abs().amax(-1)
    assert err.max() < (3e-5 if dtype == torch.float32 else 0.1), (err.argmax().item(), err.max().item())


MIXERS = [attn(4, 2, 32, 24, 41, 16)[1], attn(3, 3, 20, 12, 129, 6)[1], attn(40, 2, 128, 128, 1000, 64)[1], attn(8, 1, 96, 112, 128, 96)[1], attn(16, 1, 192, 128, 64, 8)[1],
          attn(2, 2, 64, 200, 77, 64)[1], attn(6, 2, 256, 256, 50, 128)[1], attn(5, 5, 64, 64, 0, 0)[1], attn(2, 1, 300, 264, 90, 20)[1]]


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("mx", MIXERS, ids=lambda m: "-".join(str(m[k]) for k in ("heads", "kv_heads", "dim", "vdim")) + f"-c{m['mask']['size']}")
def test_grouped_attention(mx, where):
    """Decoded tokens, prompt chunks (one and several 128- and 256-row blocks), short portions, and all of them in one batch."""
    _check(mx, [1, 2, 40, 41, 42, 128, 129, 300, 1100], [1] * 9, where)
    _check(mx, [700], [700], where, seed=1)
    _check(mx, [17, 300, 1100, 129, 600], [17, 257, 130, 128, 18], where, seed=2)
    _check(mx, [500, 260, 90, 1030, 33], [1, 200, 2, 300, 16], where, seed=3)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("mx", [attn(4, 2, 32, 24, 41, 16, scale=1.0)[1], attn(9, 3, 128, 128, 130, 64, scale=0.5)[1], attn(2, 1, 24, 40, 257, 24, scale=1.0)[1]],
                         ids=["c41", "c130", "c257"])
def test_far_keys_stand_out(mx, where):
    """One key carries nearly all of a query's weight: at the chunk's first position, one before it (unseen), at page borders and far
    back, for decoded rows and for rows of a portion."""
    C = mx["mask"]["size"]
    n = 3 * C + 300
    for news in (1, 2, 16, 17, 300) if where[0] == "cuda" else (1, 300):
        for i in sorted({0, news // 2, news - 1}):
            at = n - news + i                                       # position of the query
            for j in {at, at - at % C, at - at % C - 1, at - C // 2, (at // PAGE) * PAGE, (at // PAGE) * PAGE - 1, at - C - 100}:
                if 0 <= j <= at:
                    _check(mx, [n, 200], [news, 1], where, seed=j, strong=[(0, i, j, 30.0)])


@pytest.mark.parametrize("where", DEVICES)
def test_many_decoded_rows(where):
    """More rows than one call of the decode kernel takes."""
    n = 40 if where[0] == "cuda" else 3
    _check(attn(2, 1, 32, 32, 50, 16)[1], [200 + b for b in range(n)], [16] * n, where)


def _gla_case(mx, parts, device, dtype, rank=16, seed=0, z_shift=0.0, z_scale=1.0):
    """Requests cut into ``parts`` (lists of portion lengths, one step each), in state slots handed out in reverse; a step is one batch."""
    g = torch.Generator().manual_seed(seed)
    H, D, V = mx["heads"], mx["dim"], mx["vdim"]
    r16 = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    a2, a2b, nw = (r16(H * D, rank) * z_scale * rank ** -0.5).to(torch.bfloat16), (r16(H * D) * 0.5 + z_shift).to(torch.bfloat16), (1 + 0.2 * r16(V)).to(torch.bfloat16)
    lens = [sum(p) for p in parts]
    x = [dict(q=r16(n, H * D), k=r16(n, H * D), v=r16(n, H * V), g=r16(n, H * V), a=r16(n, rank)) for n in lens]
    want = []
    for t in x:
        n = t["q"].shape[0]
        z = O.linear(a2.double(), t["a"].double()) + a2b.double()
        rs = lambda m, d: m.double().reshape(n, H, d)
        o, _ = O.gla_recurrence(rs(t["q"], D) * D ** -0.5, rs(t["k"], D), rs(t["v"], V), O.gla_log_decay(rs(z, D), mx["tau"]), torch.zeros(H, D, V, dtype=torch.float64))
        want.append(O.gla_finish(o, t["g"].double(), nw.double(), 1e-5))
    to = lambda t: t.to(device, dtype)
    z = lambda n: torch.zeros(n, 16, dtype=dtype, device=device)
    w, _ = GLA.build(GLASpec(H, D, V, mx["tau"]), z(H * D), z(H * D), z(H * V), z(H * V), z(rank), to(a2), to(a2b), to(nw))
    state = torch.zeros((len(parts) + 1, H, D, V), device=device)
    state[-1] = 5.0                                                   # a slot nobody uses
    done, got = [0] * len(parts), [[] for _ in parts]
    for s in range(max(len(p) for p in parts)):
        reqs = [b for b in range(len(parts)) if s < len(parts[b]) and parts[b][s]]
        cu, rows = [0], []
        for b in reqs:
            n = parts[b][s]
            cu.append(cu[-1] + n)
            row = torch.zeros(n, (w.cols[-1] + rank + 31) // 32 * 32)
            for key, c in zip("qkvga", w.cols):
                m = x[b][key][done[b]:done[b] + n]
                row[:, c:c + m.shape[1]] = m.float()
            rows.append(row)
            done[b] += n
        slots = [len(parts) - 1 - b for b in reqs]
        i32 = lambda t: torch.tensor(t, dtype=torch.int32, device=device)
        fb = ForwardBatch(ids=None, positions=None, slots=None, page_table=i32([[0]]), kv_lens=None, cu_q=i32(cu), cu_q_host=cu, is_decode=cu == list(range(len(cu))),
                          state_slots=i32(slots), state_slots_host=slots)
        y = GLA.mix(w, to(torch.cat(rows)), fb, state, 1e-5).cpu().double()
        for i, b in enumerate(reqs):
            got[b].append(y[cu[i]:cu[i + 1]])
    assert (state[-1] == 5.0).all()
    return torch.cat([torch.cat(t) for t in got]), torch.cat(want)


def _check_gla(mx, parts, where, **kw):
    device, dtype = where
    got, want = _gla_case(mx, parts, device, dtype, **kw)
    assert torch.isfinite(got).all()
    err = (got - want).abs().amax(-1)
    assert err.max() < (1e-4 if dtype == torch.float32 else 0.08) * (1 + want.abs().amax(-1)[err.argmax()]), (err.argmax().item(), err.max().item())


GLAS = [(gla(3, 24, 40, 8.0)[1], 16), (gla(1, 8, 8, 1.0)[1], 1), (gla(2, 20, 12, 4.0)[1], 5), (gla(4, 128, 128, 16.0)[1], 16), (gla(2, 64, 192, 16.0)[1], 64),
        (gla(1, 256, 256, 12.0)[1], 24), (gla(2, 96, 64, 16.0)[1], 80)]


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("mx,rank", GLAS, ids=lambda v: "-".join(str(x) for x in v.values()) if isinstance(v, dict) else f"r{v}")
def test_gated_linear_attention(mx, rank, where):
    """Whole prompts, portions of every kind (chunk borders just missed), single tokens, and batches of them."""
    n = 1 if where[0] == "cpu" else 3
    _check_gla(mx, [[65 * n]], where, rank=rank)
    _check_gla(mx, [[1] * 12, [1] * 12, [1] * 9], where, rank=rank, seed=1)
    _check_gla(mx, [[63, 1, 2, 64, 1], [2, 2, 70, 1, 1], [1, 1, 1, 1, 1], [64, 65, 0, 3, 17], [16 * n, 1, 15, 33, 2]], where, rank=rank, seed=2)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("shift,scale", [(-90.0, 1.0), (-6.0, 6.0), (60.0, 1.0), (0.0, 40.0)])
def test_decay_extremes(shift, scale, where):
    """Channels that forget within a token beside channels that never do: nothing overflows and nothing is lost."""
    _check_gla(gla(2, 32, 24, 1.0)[1], [[130, 1, 1, 40], [7, 64, 1, 1]], where, z_shift=shift, z_scale=scale)


@pytest.mark.parametrize("where", DEVICES)
def test_first_token_survives(where):
    """With decays of almost one, the first token's value is still read after many chunks (and a late state keeps its precision)."""
    device, dtype = where
    for parts in ([[300]], [[2, 150, 100, 48]], [[64] * 4 + [1] * 44]):
        _check_gla(gla(1, 16, 8, 16.0)[1], parts, where, z_shift=9.0, z_scale=0.1, seed=4)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("shape", [(6, 3, 48, 160), (9, 1, 112, 256), (64, 6, 64, 384), (1, 1, 8, 72), (40, 40, 16, 64)], ids=str)
@pytest.mark.parametrize("rows", [1, 7, 300, 900])
def test_scored_experts(tmp_path, shape, rows, where):
    """Router, plan (also the one for many pairs), scaled gather, clamped experts, combine, output norm and residual (one layer)."""
    device, dtype = where
    E, top, ff, width = shape
    cfg = config([(gla(1, 8, 8, 4.0), moe(E, top, ff, 0.9))], width=width, vocab=112)
    w = O.random_weights(cfg, seed=E)
    m = load_model(save(tmp_path / "m", cfg, w), device=device, dtype=dtype)
    f = m.layers[0].mlp
    g = torch.Generator().manual_seed(rows)
    rows = rows if where[0] == "cuda" else min(rows, 7)
    x = torch.randn(rows, width, generator=g).to(torch.bfloat16)
    wd = {k: v.double() for k, v in w.items()}
    s = torch.sigmoid(x.double() @ wd["l0.mlp.router"].T).sort(dim=1, descending=True).values
    clear = (s[:, top - 1] - s[:, top] > 1e-4) if top < E else torch.ones(rows, dtype=torch.bool)
    h = x.float().to(device)
    h, y = m._mlp(f, x.to(device, dtype), h, 0, None, None, None)
    z = O.moe(x.double(), wd, "l0.mlp.", cfg["layers"][0]["mlp"])
    want = x.double() + O.rms_norm(z, wd["l0.norm2"], 1e-5)
    tol = 5e-5 if dtype == torch.float32 else 0.06
    assert clear.double().mean() > 0.9
    assert (h.cpu().double() - want)[clear].abs().max() < tol * (1 + want.abs().max())
    assert (y.cpu().double() - want)[clear].abs().max() < (tol if dtype == torch.float32 else 0.1) * (1 + want.abs().max())
    idx, sc = MOE.route_scored(f, x.to(device, dtype))
    assert idx.shape == (rows, top) and (sc.cpu().double() - s[:, :top])[clear].abs().max() < 1e-5


@pytest.mark.parametrize("where", DEVICES)
def test_clamps_show(tmp_path, where):
    """Experts whose branches mostly lie beyond the limit, on either side."""
    device, dtype = where
    cfg = config([(gla(1, 8, 8, 4.0), moe(2, 2, 64, 0.25))], width=64, vocab=32)
    w = O.random_weights(cfg, seed=3)
    for k in w:
        if k.endswith(".gate") or k.endswith(".up"):
            w[k] = w[k] * 4
    m = load_model(save(tmp_path / "m", cfg, w), device=device, dtype=dtype)
    x = torch.randn(20, 64, generator=torch.Generator().manual_seed(1)).to(torch.bfloat16)
    h, _ = m._mlp(m.layers[0].mlp, x.to(device, dtype), x.float().to(device), 0, None, None, None)
    wd = {k: v.double() for k, v in w.items()}
    want = x.double() + O.rms_norm(O.moe(x.double(), wd, "l0.mlp.", cfg["layers"][0]["mlp"]), wd["l0.norm2"], 1e-5)
    assert (h.cpu().double() - want).abs().max() < (1e-4 if dtype == torch.float32 else 0.15)


# ---------------------------------------------------------------------------------------------------
# configuration, scheduler, sampling
# ---------------------------------------------------------------------------------------------------
def test_layers_and_their_pools(models):
    cfg, w, path = models("mixed")
    eng = open_engine(path, torch.float32, 256, "cpu")
    m, pools = eng.model, eng.runner.kv.pools
    assert [type(x) for x in m.cfg.mixers] == [AttnSpec, GLASpec, AttnSpec, GLASpec, AttnSpec]
    assert pools[2][0] is pools[0][0] and pools[2][1] is pools[0][1] and pools[4][0] is not pools[0][0]
    assert pools[0][0].shape[2:] == (3, 40) and pools[0][1].shape[2:] == (3, 24) and pools[4][1].shape[2:] == (4, 72)
    assert pools[1][1].shape == (5, 3, 24, 40) and pools[3][1].shape == (5, 2, 64, 16) and pools[1][1].dtype == torch.float32
    assert m.kv_bytes_per_page() == 4 * PAGE * (3 * 64 + 4 * 136)
    assert m.linear_state_bytes_per_slot() == 4 * (3 * 24 * 40 + 2 * 64 * 16)
    assert m.layers[2].grouped.own_kv is False and m.layers[2].grouped.k_norm is None and m.layers[1].mlp.absent


def test_unknown_parts_are_refused():
    bad = []
    for change in (lambda c: c["layers"][0].update(type="something_else"), lambda c: c["layers"][1]["mlp"].update(kind="dense"),
                   lambda c: c["layers"][1]["mixer"].update(kv_from=0), lambda c: c["layers"][1]["mixer"].update(kv_from=1)):
        cfg = json.loads(json.dumps(CONFIGS["ones"]))
        change(cfg)
        with pytest.raises((NotImplementedError, ValueError)):
            from_hf_dict(cfg)
        bad.append(cfg)
    assert len(bad) == 4


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
    path = models("mixed")[2]
    m = load_model(path, device="cpu", dtype=torch.float32)
    prompts, outs = [prompt("mixed", 9, 5) * 4, [7, 8, 9] * 10], []
    for spec in ("", "ngram"):
        eng = LLMEngine(m, EngineConfig(max_batch=2, max_context=256, speculative=spec), num_pages=8)
        outs.append(eng.generate(prompts, GenerationConfig(max_new_tokens=12, ignore_eos=True)))
    assert outs[0] == outs[1]


def test_layers_without_pages(tmp_path):
    """A stack of recurrent layers only: no page pools, the scheduler runs on state slots."""
    cfg = config([(gla(2, 16, 16, 4.0), moe(2, 1, 16, 1.0)), (gla(1, 24, 8, 2.0), None)], width=64, vocab=64)
    w = O.random_weights(cfg, seed=1)
    m = load_model(save(tmp_path / "m", cfg, w), device="cpu", dtype=torch.float32)
    eng = LLMEngine(m, EngineConfig(max_batch=2, max_context=256, max_tokens=512))
    toks = list(range(20))
    out = eng.generate([toks, toks[:3]], GenerationConfig(max_new_tokens=3, ignore_eos=True))
    logits = O.forward(cfg, w, toks + out[0][:-1])[19:]
    assert [x.argmax().item() for x in logits] == out[0]


def test_context_ends_with_the_position_table(models):
    path = models("ones")[2]
    eng = LLMEngine(load_model(path, device="cpu", dtype=torch.float32), EngineConfig(max_batch=2, max_context=4096), num_pages=16)
    assert eng.cfg.max_context == 640
    out = eng.generate([prompt("ones", 636, 1)], GenerationConfig(max_new_tokens=50, ignore_eos=True))
    assert 1 <= len(out[0]) <= 5


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
    seq = toks + out
    want = O.forward(cfg, w, seq[:-1])[len(toks) - 1:]
    assert len(out) == 4 and all((want[k].max() - want[k][t]) < 0.1 for k, t in enumerate(out))
    tiny = random_init(preset("tiny-vilulorn"), "cpu", torch.float32)
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
