"""Nasipel (latent attention with query latents, rotated parts and head gates; sigmoid-weighted attention over rotated values; real-gated
linear recurrent units; gated sub-layers side by side, experts chosen by corrected sigmoid scores) against its plain statement.

Every case builds a small random model of its own.  The CPU runs use the framework's PyTorch operator definitions (scheduling,
cache, loading and the model itself); the GPU runs the kernels, in float32 and bfloat16.
"""
import json

import pytest
import torch

from . import listed_common as LC
from . import nasipel_oracle as O
from .listed_common import DEVICES, PAGE, assert_close, few_threads, portions, save  # noqa: F401
from fastllm_b200.engine import EngineConfig, GenerationConfig, LLMEngine
from fastllm_b200.engine.replay import Replay, open_engine
from fastllm_b200.loader.hf import load_model
from fastllm_b200.models.config import AttnSpec, LatentSpec, RGLRUSpec, from_hf_dict
from fastllm_b200.models.decoder import ForwardBatch
from fastllm_b200.ops import attention as A
from fastllm_b200.ops import basic as B
from fastllm_b200.ops import grouped as GR
from fastllm_b200.ops import latent as LA
from fastllm_b200.ops import moe as MOE
from fastllm_b200.ops import rglru as RG
from fastllm_b200.ops import stream32 as S
from fastllm_b200.ops.quant import LinearWeight

gpu = pytest.mark.gpu


def attn(heads, kv, dim, vdim, rot, cap=20.0, scale=None, base=1e4):
    m = {"heads": heads, "kv_heads": kv, "dim": dim, "vdim": vdim, "scale": scale or 1.1 * dim ** -0.5, "rot": {"base": base, "dims": rot}}
    return "attention", dict(m, softcap=cap) if cap else m


def latent(heads, dim, rot, vdim, q_rank, kv_rank, yarn=None, base=2e4, scale=None):
    r = {"base": base, "dims": rot}
    if yarn:
        r["scaling"] = dict(zip(("factor", "original", "fast", "slow"), yarn))
    return "latent_attention", {"heads": heads, "dim": dim, "rot_dim": rot, "vdim": vdim, "q_rank": q_rank, "kv_rank": kv_rank, "scale": scale or (dim + rot) ** -0.5, "rot": r}


def unit(width, blocks, conv):
    return "rglru", {"width": width, "blocks": blocks, "conv": conv}


def moe(experts, top, ff, groups=None, scale=None):
    r = {"experts": experts, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    if scale:
        r["scale"] = scale
    return {"kind": "moe", "expert": {"ff": ff}, "router": r}


def config(layers, width=160, vocab=304, eps=1e-5):
    return {"architecture": "Nasipel", "vocab": vocab, "width": width, "norm": {"eps": eps}, "max_position_embeddings": 4096, "layers": [{"type": t, "mixer": m, "mlp": f} for (t, m), f in layers]}


YARN = (6.0, 100, 16.0, 1.0)
CONFIGS = {
    # every expert is taken (no close calls in 16 bits); one layer without feed-forward
    "mixed": config([(unit(96, 3, 4), moe(3, 3, 48, scale=1.7)), (latent(3, 40, 16, 24, 56, 72, YARN), None), (attn(6, 3, 40, 24, 16), moe(2, 2, 112, scale=0.6)),
                     (latent(4, 32, 32, 64, 64, 128), moe(3, 3, 64)), (unit(128, 1, 2), moe(2, 2, 40))]),
    # nothing is a multiple of anything the kernels tile
    "odd": config([(attn(3, 1, 20, 12, 6, cap=7.0), moe(3, 3, 75, scale=1.3)), (unit(60, 3, 5), moe(2, 2, 31)), (latent(3, 20, 6, 12, 30, 33, (3.5, 40, 8.0, 2.0)), moe(3, 3, 30)),
                   (attn(5, 5, 18, 14, 18), None), (unit(13, 13, 3), moe(2, 2, 9))], width=148, vocab=331, eps=1e-4),
    # heads of a served size: sixteen query heads per key head, whole tensor-core tiles, wide blocks
    "wide": config([(latent(18, 128, 64, 128, 192, 512, (8.0, 64, 32.0, 1.0)), moe(2, 2, 128)), (attn(32, 2, 128, 128, 128, cap=40.0), moe(4, 4, 64, scale=2.5)), (unit(512, 2, 4), None),
                    (attn(24, 1, 192, 128, 64), moe(2, 2, 64)), (unit(256, 4, 3), moe(2, 2, 64))], width=256, vocab=512),
    # one of everything
    "ones": config([(attn(1, 1, 8, 8, 2), moe(1, 1, 8, (1, 1))), (unit(8, 1, 1), moe(1, 1, 8)), (latent(1, 8, 2, 8, 8, 8), moe(1, 1, 8))], width=64, vocab=64),
    # none of the optional parts
    "bare": config([(unit(32, 2, 2), None), (attn(4, 2, 32, 32, 32, cap=None), moe(2, 2, 40)), (latent(2, 32, 16, 32, 48, 64), None)], width=128, vocab=200),
    # experts are chosen within their best groups
    "routed": config([(attn(4, 2, 32, 32, 16), moe(40, 3, 64, (8, 3), 2.0)), (unit(64, 2, 4), moe(6, 1, 40, (3, 1))), (latent(2, 32, 16, 32, 48, 64), moe(12, 4, 32, (6, 4)))],
                     width=128, vocab=256),
}
OVER = {"routed": 0.5}
_CACHE: dict = {}


def weights(name):
    if name not in _CACHE:
        _CACHE[name] = O.random_weights(CONFIGS[name], seed=len(name))
    return _CACHE[name]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, weights, checkpoint folder); the folders are written once."""
    root, out = tmp_path_factory.mktemp("nasipel"), {}

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
    """From the first token on, across page borders."""
    n = 20 if where[0] == "cpu" else 300
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
    rp = Replay(open_engine(path, dtype, 8 * PAGE, device))
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
# mechanisms alone: norms, gates, rotations
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("width", [64, 148, 75, 2080])
def test_gated_join(width, where):
    """Embedding; mixer and experts behind their gates, each alone and both; one or two norms, with and without the mean."""
    device, dtype = where
    g = torch.Generator().manual_seed(width)
    r16 = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    T, top = 6, 3
    table, w1, w2, y1, g1, ys = r16(50, width), r16(width), r16(width), r16(T, width), r16(T, width + 8), r16(T * top + 5, width)
    pos = torch.randperm(T * top, generator=g).view(T, top).int()
    pos[1, 2] = -1                                                    # a pair that is held elsewhere
    wts, g2 = torch.rand(T, top, generator=g), torch.randn(T, width + 12, generator=g)
    ids, h0 = torch.randint(0, 50, (T,), generator=g), 3 + torch.randn(T, width, generator=g)
    to = lambda t: t.to(device, dtype)
    tol = 2e-5 if dtype == torch.float32 else 0.03
    dense = (ys.double()[pos.long().clamp(min=0)] * torch.where(pos >= 0, wts, 0.0).double()[..., None]).sum(1)
    for center in (True, False):
        norm = O.layer_norm if center else O.rms_norm
        for embed in (None, (to(table), ids.int().to(device))):
            for mixer in (None, (to(y1), to(g1)[:, 8:])):
                for ff, out in ((None, 0), ((to(ys), pos.to(device), wts.to(device), g2.to(device)[:, :width]), dense),
                                ((to(ys)[:T], None, None, g2.to(device)[:, :width]), ys[:T].double())):
                    for second in (None, to(w2)):
                        h = h0.clone().to(device)
                        a, b = S.gated_join(h, mixer, ff, to(w1), second, 1e-4, dtype, center, embed)
                        want = (table[ids] if embed else h0).double()
                        if mixer:
                            want = want + torch.sigmoid(g1[:, 8:].double()) * y1.double()
                        if ff:
                            want = want + torch.sigmoid(g2[:, :width].double()) * out
                        assert (h.cpu().double() - want).abs().max() < 2e-5
                        for got, w in ((a, w1), (b, w2)):
                            if got is None:
                                assert second is None
                                continue
                            ref = norm(want, w.double(), 1e-4)
                            assert got.dtype == dtype and (got.cpu().double() - ref).abs().max() < tol * (1 + ref.abs().max())


@pytest.mark.parametrize("where", DEVICES)
def test_norm_of_a_far_mean(where):
    """The variance is that of the deviations: rows far from zero keep their precision."""
    device, dtype = where
    h = (1000.0 + torch.randn(5, 256, generator=torch.Generator().manual_seed(1))).to(device)
    a, _ = S.gated_join(h, None, None, torch.ones(256, device=device, dtype=dtype), None, 1e-6, dtype)
    want = O.layer_norm(h.cpu().double(), torch.ones(256).double(), 1e-6)
    assert (a.cpu().double() - want).abs().max() < (1e-3 if dtype == torch.float32 else 0.03)


@pytest.mark.parametrize("dims,base,sc", [(32, 5e4, (8.0, 1024, 32.0, 1.0)), (64, 5e5, (40.0, 4096, 32.0, 1.0)), (16, 1e4, (4.0, 64, 32.0, 1.0)), (8, 1e4, (2.5, 77, 3.0, 3.0)),
                                          (32, 1e4, (0.5, 50, 64.0, 2.0)), (2, 1e3, (4.0, 100000, 1.0, 1.0)), (4, 20.0, (3.0, 1000000, 2.0, 1.0))], ids=str)
def test_scaled_frequencies(dims, base, sc):
    """Tables of the scaled rotation, ramps that are cut off at either end or have no width, positions far beyond the original length."""
    spec = from_hf_dict(config([(latent(2, 16, dims, 16, 16, 16, sc, base), None)])).mixers[0]
    cos, sin = A.build_rope_tables(dims, 3000, spec.rope["theta"], spec.rope["scaling"])
    freqs, mag = O.yarn_freqs(dims, base, dict(zip(("factor", "original", "fast", "slow"), sc)))
    for p in (0, 1, 77, 2999):
        a = torch.tensor([p * f for f in freqs], dtype=torch.float64)
        assert (cos[p].double() - mag * a.cos()).abs().max() < 2e-7 * mag and (sin[p].double() - mag * a.sin()).abs().max() < 2e-7 * mag


# ---------------------------------------------------------------------------------------------------
# attention with sigmoid weights and rotated values
# ---------------------------------------------------------------------------------------------------
def _tables(lens, dev, g):
    """Page table [requests, pages] in a shuffled order, and the number of pages."""
    npg = [(n + PAGE - 1) // PAGE for n in lens]
    order = torch.randperm(sum(npg), generator=g).tolist()
    table = torch.zeros((len(lens), max(npg)), dtype=torch.int32)
    for b in range(len(lens)):
        for i in range(npg[b]):
            table[b, i] = order.pop()
    return table, sum(npg)


def _batch(table, first, last, device):
    """Tokens [first[b], last[b]) of every request."""
    cu, pos, slots = [0], [], []
    for b in range(len(last)):
        p = torch.arange(first[b], last[b])
        cu.append(cu[-1] + len(p))
        pos.append(p)
        slots.append(table[b][p // PAGE].long() * PAGE + p % PAGE)
    i32 = lambda t: torch.as_tensor(t).to(torch.int32).to(device)
    return ForwardBatch(ids=i32(torch.cat(pos)), positions=i32(torch.cat(pos)), slots=i32(torch.cat(slots)), page_table=table.to(device), kv_lens=i32(last), cu_q=i32(cu),
                        cu_q_host=cu, is_decode=all(cu[i + 1] - cu[i] == 1 for i in range(len(last))), kv_lens_host=list(last))


def _case(mx, lens, news, device, dtype, seed=0, strong=(), bias=None):
    """Cached keys and values of requests with ``lens`` tokens, of which the last ``news`` are this batch's, through ``post`` and
    ``attention``.  ``strong``: (request, query index, key index): that query points at that key, in every head."""
    g = torch.Generator().manual_seed(seed)
    H, G, D, V, rot = mx["heads"], mx["kv_heads"], mx["dim"], mx["vdim"], mx["rot"]
    r16 = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    k, v = [r16(n, G, D) for n in lens], [r16(n, G, V) for n in lens]
    q = [r16(n, H, D) for n in news]
    bias = -3.0 + torch.randn(H, generator=g) if bias is None else bias
    eps, pos = 1e-5, [torch.arange(n) for n in lens]
    fr, fv = O.plain_freqs(rot["dims"], rot["base"]), O.plain_freqs(V, rot["base"])
    kr = [O.unit_rms(O.turn(k[b].double(), pos[b], fr, True), eps) for b in range(len(lens))]
    for b, i, j in strong:
        at = lens[b] - news[b] + i
        seen = O.turn(kr[b][j:j + 1], torch.tensor([at]), fr, True, sign=-1.0)[0]       # the key seen from the query's position
        for h in range(H):
            q[b][i, h] = seen[h // (H // G)].to(torch.bfloat16)
    want = []
    for b, (n, m) in enumerate(zip(lens, news)):
        qr = O.unit_rms(O.turn(q[b].double(), pos[b][n - m:], fr, True), eps)
        want.append(O.turn(O.sigmoid_attention(qr, kr[b], O.turn(v[b].double(), pos[b], fv, True), mx, bias), pos[b][n - m:], fv, True, sign=-1.0))
    spec = from_hf_dict(config([(("attention", mx), None)])).mixers[0]
    z = lambda n: torch.zeros(n, 16, dtype=dtype, device=device)
    w, _ = GR.build(spec, z(H * D), z(G * D), z(G * V), None, None, None, score_bias=bias.to(device))
    cos, sin = A.build_rope_tables(rot["dims"], 4096, rot["base"], None, device)
    w.turn = A.build_rope_tables(V, 4096, rot["base"], None, device)
    order = GR.value_order(spec)
    table, pages = _tables(lens, device, g)
    kp = torch.full((pages, PAGE, G, w.dp), 3.0, dtype=dtype, device=device)                 # pages start dirty
    vp = torch.full((pages, PAGE, G, w.vp), -2.0, dtype=dtype, device=device)

    def run(first, last):
        fb, rows = _batch(table, first, last, device), []
        for b in range(len(lens)):
            row = torch.zeros(last[b] - first[b], (w.v_col + G * w.vp + 31) // 32 * 32)
            put = lambda c, x, m: row[:, c:c + x.shape[1] * m].view(len(row), x.shape[1], m)[..., :x.shape[2]].copy_(x.float())
            if last[b] == lens[b]:
                put(0, q[b], w.dp)
            put(w.k_col, k[b][first[b]:last[b]], w.dp)
            put(w.v_col, v[b][first[b]:last[b]][..., order], w.vp)
            rows.append(row)
        proj = torch.cat(rows).to(device, dtype)
        GR.post(w, proj, fb, (kp, vp), cos, sin, eps)
        return fb, proj

    if any(n > m for n, m in zip(lens, news)):                        # the earlier tokens' keys and values
        run([0] * len(lens), [n - m for n, m in zip(lens, news)])
    fb, proj = run([n - m for n, m in zip(lens, news)], lens)
    got = GR.attention(w, proj, (kp, vp), fb).cpu().double().view(-1, H, w.vp)
    assert (got[..., V:] == 0).all()
    back = torch.empty_like(order)
    back[order] = torch.arange(V)
    return got[..., :V][..., back], torch.cat(want)


def _check(mx, lens, news, where, **kw):
    device, dtype = where
    got, want = _case(mx, lens, news, device, dtype, **kw)
    err = (got - want).abs().amax((1, 2)) / (1 + want.abs().amax((1, 2)))
    assert err.max() < (5e-5 if dtype == torch.float32 else 0.04), (err.argmax().item(), err.max().item())


MIXERS = [attn(4, 2, 32, 24, 16)[1], attn(3, 1, 20, 12, 6, cap=2.0)[1], attn(40, 2, 128, 128, 128, cap=30.0)[1], attn(2, 2, 256, 192, 64)[1], attn(2, 1, 300, 264, 300)[1],
          attn(3, 3, 18, 14, 18, cap=None)[1], attn(8, 1, 96, 112, 96)[1], attn(16, 1, 192, 128, 8)[1], attn(2, 2, 64, 250, 2, cap=5.0)[1], attn(5, 5, 64, 2, 64)[1]]
_IDS = lambda m: "-".join(str(m[k]) for k in ("heads", "kv_heads", "dim", "vdim"))


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("mx", MIXERS, ids=_IDS)
def test_attention(mx, where):
    """Decoded tokens, prompt blocks (one and several 128- and 256-row blocks), short portions, and all of them in one batch."""
    if where[0] == "cpu" and mx["heads"] * mx["dim"] > 600:
        return _check(mx, [17, 300, 129], [17, 140, 1], where)
    _check(mx, [1, 2, 40, 41, 42, 128, 129, 300, 1100], [1] * 9, where)
    _check(mx, [700], [700], where, seed=1)
    _check(mx, [17, 300, 1100, 129, 600], [17, 257, 130, 128, 18], where, seed=2)
    _check(mx, [500, 260, 90, 1030, 33], [1, 200, 2, 300, 16], where, seed=3)


@pytest.mark.parametrize("where", DEVICES)
def test_far_keys_stand_out(where):
    """One key carries nearly all of the weight (the others' sigmoids are closed): the first ones, page and step borders, the query itself."""
    cpu = where[0] == "cpu"
    for mx in (attn(4, 2, 32, 24, 16, cap=None, scale=0.9)[1], attn(2, 1, 128, 64, 128, cap=30.0, scale=0.3)[1]):
        bias = torch.full((mx["heads"],), -14.0)
        for n, news in ((700, 1), (900, 300)) if cpu else ((700, 1), (700, 2), (900, 300), (640, 16)):
            for j in (0, PAGE - 1, PAGE) if cpu else (0, 1, 63, 64, PAGE - 1, PAGE, 4 * PAGE - 1, 4 * PAGE, n - news):
                device, dtype = where
                got, want = _case(mx, [n, 40], [news, 17], device, dtype, seed=j, strong=[(0, 0, j), (0, news - 1, j)], bias=bias)
                for r in (0, news - 1):
                    assert want[r].abs().max() > 0.5
                    assert (got - want)[r].abs().max() < (1e-4 if dtype == torch.float32 else 0.06), (n, news, j, r)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("level", [-60.0, -20.0, 0.0, 30.0])
def test_weights_do_not_compete(level, where):
    """Sigmoids that are shut, open and in between, for one key and for many: their sum is not normalised."""
    mx = attn(6, 2, 32, 24, 16, cap=8.0)[1]
    bias = level + torch.tensor([0.0, 1.0, -1.0, 2.0, -2.0, 0.5])
    for lens, news in (([1, 2, 200, 520], [1, 1, 1, 1]), ([1, 200, 520], [1, 200, 300])):
        device, dtype = where
        got, want = _case(mx, lens, news, device, dtype, bias=bias)
        floor = want.abs().amax()
        if level > -60:
            assert (got - want).abs().max() < (5e-5 if dtype == torch.float32 else 0.02) * floor
        else:
            assert got.abs().max() < 1e-14                             # (a clamp keeps tiny weights finite)


@pytest.mark.parametrize("where", DEVICES)
def test_soft_cap_shows(where):
    """Scores far beyond the cap on either side: many keys end up alike."""
    _check(attn(4, 2, 32, 24, 16, cap=1.5, scale=2.0)[1], [300, 70], [300, 1], where)


@pytest.mark.parametrize("where", DEVICES)
def test_many_decoded_rows(where):
    """More rows than one call of the decode kernel takes."""
    n = 40 if where[0] == "cuda" else 3
    _check(attn(2, 1, 32, 32, 16)[1], [200 + b for b in range(n)], [16] * n, where)


# ---------------------------------------------------------------------------------------------------
# latent attention
# ---------------------------------------------------------------------------------------------------
def _latent_case(mx, lens, news, device, dtype, seed=0, strong=(), gain=1.0, direct=False):
    """``post`` and ``attention`` of one layer over cached rows.  ``strong``: (request, query index, key index): the rotated parts of that
    query point at that key.  ``direct``: queries without a latent of their own."""
    g = torch.Generator().manual_seed(seed)
    H, D, R, V, K, Q = (mx[k] for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank", "q_rank"))
    r16 = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    m16 = lambda n, k: (torch.randn(n, k, generator=g) * k ** -0.5).to(torch.bfloat16)
    uq, uk, uv, qn, kn = m16(H * (D + R), Q), m16(H * D, K), (1.5 * m16(H * V, K).float()).to(torch.bfloat16), r16(Q), r16(K)
    rot, eps = mx["rot"], 1e-5
    fr, mag = O.yarn_freqs(R, rot["base"], rot["scaling"]) if rot.get("scaling") else (O.plain_freqs(R, rot["base"]), 1.0)
    cq, ckv, gate = [r16(n, H * (D + R) if direct else Q) for n in news], [r16(n, K + R) for n in lens], [r16(n, H) for n in news]
    cq = [c * 0.3 for c in cq] if direct else cq
    for b, i, j in strong:                                            # (needs direct queries)
        at = lens[b] - news[b] + i
        key = O.turn(ckv[b][j:j + 1, K:].double().view(1, 1, R), torch.tensor([at - j]), fr, False, sign=-1.0)[0, 0]
        cq[b].view(news[b], H, D + R)[i, :, D:] = (gain * key / key.norm() / mag ** 2).to(torch.bfloat16)
    want = []
    for b, (n, m) in enumerate(zip(lens, news)):
        pos = torch.arange(n)
        q = (cq[b].double() if direct else O.linear(uq.double(), O.rms_norm(cq[b].double(), qn.double(), eps))).reshape(m, H, D + R)
        c = O.rms_norm(ckv[b][:, :K].double(), kn.double(), eps)
        qr, kr = O.turn(q[..., D:], pos[n - m:], fr, False, mag=mag), O.turn(ckv[b][:, K:].double().view(n, 1, R), pos, fr, False, mag=mag)[:, 0]
        k, v = O.linear(uk.double(), c).view(n, H, D), O.linear(uv.double(), c).view(n, H, V)
        see = pos[None, :] <= pos[n - m:, None]
        out = []
        for h in range(H):
            s = (q[:, h, :D] @ k[:, h].T + qr[:, h] @ kr.T) * mx["scale"]
            out.append(torch.softmax(s.masked_fill(~see, float("-inf")), -1) @ v[:, h])
        want.append(torch.stack(out, 1) * torch.sigmoid(gate[b].double())[..., None])
    to = lambda t: t.to(device, dtype)
    spec = from_hf_dict(config([(("latent_attention", mx), None)])).mixers[0]
    zero = lambda n: torch.zeros(n, 16, dtype=dtype, device=device)
    if direct:
        spec.q_rank = 0
        w, _, _ = LA.build(spec, zero(H * (D + R)), zero(H), zero(K + R), to(kn), to(uk), to(uv))
    else:
        w, _, up = LA.build(spec, zero(Q), zero(H), zero(K + R), to(kn), to(uk), to(uv), to(uq), to(qn))
        w.q_up = LinearWeight.from_dense(up, act_dtype=dtype)
        w.q_up.exact32 = dtype == torch.float32
    rope = A.build_rope_tables(R, 4096, rot["base"], spec.rope["scaling"], device)
    table, pages = _tables(lens, device, g)
    pool = torch.full((pages + 1, PAGE, 1, w.ld), 2.0, dtype=dtype, device=device)           # pages start dirty

    def run(first, last):
        fb, rows = _batch(table, first, last, device), []
        for b in range(len(lens)):
            row = torch.zeros(last[b] - first[b], (w.more_col + 31) // 32 * 32)
            if last[b] == lens[b]:
                if direct:
                    h = cq[b].float().view(-1, H, D + R)
                    row[:, :H * w.hd].view(-1, H, w.hd)[..., :D] = h[..., :D]
                    row[:, :H * w.hd].view(-1, H, w.hd)[..., w.dim:w.dim + R] = h[..., D:]
                else:
                    row[:, :Q] = cq[b].float()
                row[:, w.gate_col:w.gate_col + H] = gate[b].float()
            row[:, w.latent_col:w.latent_col + K] = ckv[b][first[b]:last[b], :K].float()
            row[:, w.rot_col:w.rot_col + R] = ckv[b][first[b]:last[b], K:].float()
            rows.append(row)
        proj = to(torch.cat(rows))
        return fb, proj, *LA.post(w, proj, fb, pool, rope, eps)

    if any(n > m for n, m in zip(lens, news)):
        run([0] * len(lens), [n - m for n, m in zip(lens, news)])
    fb, proj, q, hg = run([n - m for n, m in zip(lens, news)], lens)
    got = LA.attention(w, proj, pool, fb, q, hg, rope).cpu().double().view(-1, H, w.vdim)
    return got[..., :V], torch.cat(want)


def _check_latent(mx, lens, news, where, **kw):
    device, dtype = where
    got, want = _latent_case(mx, lens, news, device, dtype, **kw)
    err = (got - want).abs().amax((1, 2)) / (1 + want.abs().amax((1, 2)))
    assert err.max() < (5e-5 if dtype == torch.float32 else 0.04), (err.argmax().item(), err.max().item())


LATENTS = [latent(3, 40, 16, 24, 56, 72, YARN)[1], latent(2, 20, 6, 12, 30, 33, (3.5, 40, 8.0, 2.0))[1], latent(16, 128, 64, 128, 96, 512, (8.0, 64, 32.0, 1.0))[1], latent(40, 64, 32, 48, 64, 64)[1],
           latent(2, 128, 64, 192, 64, 448)[1], latent(2, 64, 128, 64, 64, 500)[1], latent(1, 8, 2, 8, 8, 8)[1], latent(2, 32, 24, 32, 40, 576)[1], latent(2, 200, 72, 40, 24, 130)[1]]


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("mx", LATENTS, ids=lambda m: "-".join(str(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank")))
def test_latent_attention(mx, where):
    if where[0] == "cpu" and mx["heads"] * mx["dim"] > 600:
        return _check_latent(mx, [17, 300, 129], [17, 140, 1], where)
    _check_latent(mx, [1, 2, 40, 128, 129, 300, 1100], [1] * 7, where)
    _check_latent(mx, [600], [600], where, seed=1)
    _check_latent(mx, [17, 300, 900, 129], [17, 257, 130, 128], where, seed=2)
    _check_latent(mx, [500, 260, 90, 700, 33], [1, 200, 2, 300, 16], where, seed=3)
    _check_latent(mx, [260, 300, 40], [1, 270, 16], where, seed=4, direct=True)


@pytest.mark.parametrize("where", DEVICES)
def test_far_latent_keys_stand_out(where):
    """The shared rotated part alone picks one key out of hundreds, at any distance."""
    device, dtype = where
    for mx in (latent(2, 32, 32, 24, 16, 64, YARN, scale=1.0)[1], latent(2, 64, 64, 64, 16, 128, scale=1.0)[1]):
        for n, news in ((700, 1), (900, 300)) if device == "cpu" else ((700, 1), (700, 2), (900, 300), (640, 16)):
            for j in (0, PAGE - 1, PAGE) if device == "cpu" else (0, 1, 63, 64, PAGE - 1, PAGE, 4 * PAGE - 1, n - news):
                got, want = _latent_case(mx, [n, 40], [news, 17], device, dtype, seed=j, direct=True, strong=[(0, 0, j), (0, news - 1, j)], gain=12.0)
                assert (got - want)[[0, news - 1]].abs().max() < (1e-4 if dtype == torch.float32 else 0.15), (n, news, j)


# ---------------------------------------------------------------------------------------------------
# real-gated linear recurrent unit
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("shape", [(3, 2, 64, 64), (300, 3, 128, 64), (700, 2, 512, 256), (5, 4, 40, 20), (270, 1, 24, 12), (600, 5, 48, 24)], ids=str)
def test_block_products(shape, where):
    device, dtype = where
    M, blocks, N, K = shape
    g = torch.Generator().manual_seed(N)
    x, w = torch.randn(M, blocks * K, generator=g).to(torch.bfloat16), (torch.randn(blocks, N, K, generator=g) * K ** -0.5).to(torch.bfloat16)
    got = B.linear_blocks(x.to(device, dtype), w.to(device, dtype))
    want = torch.cat([O.linear(w[b].double(), x.double()[:, b * K:(b + 1) * K]) for b in range(blocks)], dim=1)
    assert got.dtype == torch.float32 and (got.cpu().double() - want).abs().max() < 2e-5 * (1 + want.abs().max())


def _unit_case(mx, parts, device, dtype, seed=0, lam=None, r_bias=0.0):
    """Requests cut into ``parts`` (lists of portion lengths, one step each), in state slots handed out in reverse; a step is one batch."""
    g = torch.Generator().manual_seed(seed)
    W, Bn, K = mx["width"], mx["blocks"], mx["conv"]
    n = W // Bn
    r16 = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    conv, conv_b, ra, ri = r16(W, K), r16(W) * 0.3, (r16(Bn, n, n) * n ** -0.5).to(torch.bfloat16), (r16(Bn, n, n) * n ** -0.5).to(torch.bfloat16)
    ra_b, ri_b = (r16(Bn, n) * 0.5 + r_bias).to(torch.bfloat16), (r16(Bn, n) * 0.5).to(torch.bfloat16)
    lam = torch.linspace(-8.0, 1.0, W).to(torch.bfloat16) if lam is None else torch.full((W,), lam).to(torch.bfloat16)
    lens = [sum(p) for p in parts]
    y, x = [r16(m, W) for m in lens], [r16(m, W) for m in lens]
    want = []
    for yy, xx in zip(y, x):
        u = O.causal_conv(xx.double(), conv, conv_b)
        want.append(O.rglru_recurrence(u, O.block_gate(u, ra, ra_b), O.block_gate(u, ri, ri_b), lam)[0] * O.gelu_tanh(yy.double()))
    to = lambda t: t.to(device, dtype)
    zero = torch.zeros(W, 16, dtype=dtype, device=device)
    w, _ = RG.build(RGLRUSpec(W, Bn, K), zero, zero, to(conv), to(conv_b), to(ra), to(ra_b), to(ri), to(ri_b), to(lam))
    state = (torch.zeros((len(parts) + 1, w.width, K - 1), device=device, dtype=dtype), torch.zeros((len(parts) + 1, w.width), device=device))
    for s in state:
        s[-1] = 5.0                                                   # a slot nobody uses
    wide = lambda t: torch.nn.functional.pad(t.float().view(-1, Bn, n), (0, w.part - n)).reshape(-1, w.width)
    done, got = [0] * len(parts), [[] for _ in parts]
    for s in range(max(len(p) for p in parts)):
        reqs = [b for b in range(len(parts)) if s < len(parts[b]) and parts[b][s]]
        cu, rows = [0], []
        for b in reqs:
            m = parts[b][s]
            cu.append(cu[-1] + m)
            rows.append(torch.cat([wide(y[b][done[b]:done[b] + m]), wide(x[b][done[b]:done[b] + m]), torch.full((m, 16), 9.0)], dim=1))
            done[b] += m
        slots = [len(parts) - 1 - b for b in reqs]
        i32 = lambda t: torch.tensor(t, dtype=torch.int32, device=device)
        fb = ForwardBatch(ids=None, positions=None, slots=None, page_table=i32([[0]]), kv_lens=None, cu_q=i32(cu), cu_q_host=cu, is_decode=cu == list(range(len(cu))),
                          state_slots=i32(slots), state_slots_host=slots)
        out = RG.mix(w, to(torch.cat(rows)), fb, state).cpu().double().view(-1, Bn, w.part)
        assert (out[..., n:] == 0).all()
        for i, b in enumerate(reqs):
            got[b].append(out[cu[i]:cu[i + 1], :, :n].reshape(-1, W))
    assert all((s[-1] == 5.0).all() for s in state)
    return torch.cat([torch.cat(t) for t in got]), torch.cat(want)


def _check_unit(mx, parts, where, **kw):
    device, dtype = where
    got, want = _unit_case(mx, parts, device, dtype, **kw)
    assert torch.isfinite(got).all()
    err = (got - want).abs().amax(-1) / (1 + want.abs().amax(-1))
    assert err.max() < (5e-5 if dtype == torch.float32 else 0.04), (err.argmax().item(), err.max().item())


UNITS = [unit(96, 3, 4)[1], unit(8, 1, 1)[1], unit(60, 3, 5)[1], unit(13, 13, 3)[1], unit(512, 2, 4)[1], unit(256, 4, 2)[1], unit(300, 1, 3)[1], unit(128, 2, 9)[1]]


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("mx", UNITS, ids=lambda v: "-".join(str(x) for x in v.values()))
def test_recurrent_unit(mx, where):
    """Whole prompts, portions of every kind (chunk borders just missed, shorter than the convolution), single tokens, and batches of them."""
    n = 1 if where[0] == "cpu" else 3
    _check_unit(mx, [[129 * n]], where)
    _check_unit(mx, [[1] * 12, [1] * 12, [1] * 9], where, seed=1)
    _check_unit(mx, [[127, 1, 2, 128, 1], [2, 2, 70, 1, 1], [1, 1, 1, 1, 1], [64, 65, 0, 3, 17], [128 * n, 1, 15, 33, 2], [257 * n, 300, 1, 2, 140]], where, seed=2)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("lam,r_bias", [(-20.0, 0.0), (-12.0, -8.0), (6.0, 4.0), (30.0, 8.0), (0.0, -40.0)])
def test_decay_extremes(lam, r_bias, where):
    """Channels that never forget (and whose inputs hardly count) and channels that forget at once."""
    _check_unit(unit(32, 2, 4)[1], [[200, 1, 1, 40], [7, 300, 1, 1]], where, lam=lam, r_bias=r_bias)


@pytest.mark.parametrize("where", DEVICES)
def test_first_token_survives(where):
    """With decays of almost one the first tokens still stand in the state after many chunks and portions."""
    for parts in ([[700]], [[2, 250, 200, 148]], [[128] * 3 + [1] * 44]):
        _check_unit(unit(16, 1, 3)[1], parts, where, lam=-9.0, seed=4)
    # and it is read: an oracle that forgets the state between the portions is far away
    got, want = _unit_case(unit(16, 1, 3)[1], [[300]], *where, lam=-5.0, seed=4)
    again, _ = _unit_case(unit(16, 1, 3)[1], [[100, 200]], *where, lam=-5.0, seed=4)
    assert (got - again).abs().max() < (1e-4 if where[1] == torch.float32 else 0.05)
    assert want[150:].abs().max() > 0.5


# ---------------------------------------------------------------------------------------------------
# experts
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("experts,top,groups", [(6, 2, (3, 1)), (40, 5, (8, 3)), (64, 6, (4, 4)), (9, 3, (9, 3)), (12, 1, (1, 1)), (16, 4, (2, 1)), (512, 8, (32, 5)), (600, 3, (3, 2)), (10, 4, (5, 2))])
def test_corrected_choice(experts, top, groups, where):
    """Groups by the sum of their two best corrected scores (negative ones among them); the weights know nothing of the correction."""
    device = where[0]
    g = torch.Generator().manual_seed(experts)
    z, corr = torch.randn(50, experts + 7, generator=g) * 3, torch.randn(experts, generator=g) - 1.0
    idx, wts = MOE.route_topk(z.to(device)[:, 4:4 + experts], corr.to(device), top, 1, True, groups[0], groups[1], 2.5)
    s = torch.sigmoid(z[:, 4:4 + experts].double())
    router = {"top": top, "groups": {"count": groups[0], "keep": groups[1]}}
    for t in range(50):
        want = O.choose(s[t] + corr.double(), router)
        assert sorted(idx[t].tolist()) == sorted(want)
        ref = s[t][idx[t].long().cpu()]
        assert (ref / ref.sum() * 2.5 - wts[t].cpu().double()).abs().max() < 3e-6


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("shape", [(6, 3, 48, 160, None, 1.5), (9, 1, 112, 256, (3, 2), None), (64, 6, 64, 384, (8, 4), 2.0), (1, 1, 8, 72, None, None), (8, 8, 200, 64, (2, 2), 0.3), (4, 2, 33, 100, (2, 2), 1.0)], ids=str)
@pytest.mark.parametrize("rows", [1, 7, 300, 900])
def test_gated_layer_with_experts(tmp_path, shape, rows, where):
    """One layer: both norms' rows in, projections with the gates beside them, router, plan, experts, the join and the last norm."""
    device, dtype = where
    E, top, ff, width, groups, scale = shape
    rows = rows if where[0] == "cuda" else min(rows, 7)
    cfg = config([(unit(16, 2, 2), moe(E, top, ff, groups, scale))], width=width, vocab=112)
    w = O.random_weights(cfg, seed=E)
    m = load_model(save(tmp_path / "m", cfg, w), device=device, dtype=dtype)
    g = torch.Generator().manual_seed(rows)
    x1, x2 = torch.randn(rows, width, generator=g).to(torch.bfloat16), torch.randn(rows, width, generator=g).to(torch.bfloat16)
    wd = {k: v.double() for k, v in w.items()}
    a, b, spec = x1.double(), x2.double(), cfg["layers"][0]
    s = torch.sigmoid(O.linear(wd["l0.mlp.router"], b)) + wd["l0.mlp.correction"]
    near = s + 1e-4 * torch.randn(s.shape, generator=g)                # rows whose choice hangs on a hair are left out
    near2 = s - 1e-4 * torch.randn(s.shape, generator=g)
    clear = torch.tensor([len({tuple(sorted(O.choose(z[t], spec["mlp"]["router"]))) for z in (s, near, near2)}) == 1 for t in range(rows)])
    i32 = lambda t: torch.tensor(t, dtype=torch.int32, device=device)
    fb = ForwardBatch(ids=i32([3] * rows), positions=i32(list(range(rows))), slots=i32([-1] * rows), page_table=i32([[0]]), kv_lens=i32([rows]), cu_q=i32([0, rows]),
                      cu_q_host=[0, rows], kv_lens_host=[rows], state_slots=i32([0]), state_slots_host=[0])
    state = (torch.zeros((1, 16, 1), device=device, dtype=dtype), torch.zeros((1, 16), device=device))
    h0 = torch.randn(rows, width, generator=g)
    h = h0.clone().to(device)
    y, none = m._gated_layer(m.layers[0], (x1.to(device, dtype), x2.to(device, dtype)), fb, state, h, 0)
    want = h0.double() + O.rglru(a, wd, "l0.mix.", spec["mixer"], 1e-5) * torch.sigmoid(O.biased(wd, "l0.rg1", a)) + O.moe(b, wd, "l0.mlp.", spec["mlp"]) * torch.sigmoid(O.biased(wd, "l0.rg2", b))
    tol = 5e-5 if dtype == torch.float32 else 0.03
    assert none is None and clear.double().mean() > 0.9
    assert (h.cpu().double() - want)[clear].abs().max() < tol * (1 + want.abs().max())
    ref = O.layer_norm(want, wd["final.norm"], 1e-5)
    assert (y.cpu().double() - ref)[clear].abs().max() < tol * (1 + ref.abs().max())


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("what", ["gate1", "gate2", "pb", "values", "unit", "cap", "yarn", "latent gate", "q norm", "decay", "conv", "correction", "scale", "mean"])
def test_every_part_counts(models, what, where, monkeypatch):
    """The reference with one part changed is far from the framework (so the other tests see it)."""
    device, dtype = where
    name = "routed" if what == "correction" else "mixed"
    cfg, w, path = models(name)
    toks = prompt(name, 190, 60)
    rp = Replay(open_engine(path, dtype, 256, device))
    got = rp.step([("a", toks, list(range(190)))], ["a"]).double()
    near = oracle(name, toks)
    cut, cw = json.loads(json.dumps(cfg)), dict(w)
    layers = cut["layers"]
    if what in ("gate1", "gate2"):
        for k in [k for k in w if k.endswith("." + {"gate1": "rg1", "gate2": "rg2"}[what])]:
            cw[k] = w[k] * 0
    elif what == "pb":
        cw["l2.mix.pb"] = w["l2.mix.pb"] + 1.0
    elif what == "values":
        plain = O.turn
        monkeypatch.setattr(O, "turn", lambda x, p, f, halves, sign=1.0, mag=1.0: plain(x, p, f, halves, sign, mag) if sign > 0 else x)
    elif what == "unit":
        monkeypatch.setattr(O, "unit_rms", lambda x, eps: x)
    elif what == "cap":
        layers[2]["mixer"]["softcap"] = 1.0
    elif what == "yarn":
        del layers[1]["mixer"]["rot"]["scaling"]
    elif what == "latent gate":
        cw["l1.mix.g"] = w["l1.mix.g"] * 0
    elif what == "q norm":
        cw["l3.mix.dq.norm"] = w["l3.mix.dq.norm"] * 0.2
    elif what == "decay":
        cw["l0.mix.lam"] = w["l0.mix.lam"] + 3
    elif what == "conv":
        cw["l0.mix.conv"] = w["l0.mix.conv"].flip(1)
    elif what == "correction":
        for k in [k for k in w if k.endswith(".correction")]:
            cw[k] = w[k] * 0
    elif what == "scale":
        layers[0]["mlp"]["router"]["scale"] = 1.0
    else:
        monkeypatch.setattr(O, "layer_norm", O.rms_norm)
        cw = {k: (v + 0.5 if k == "embed" else v) for k, v in cw.items()}
    far = O.forward(cut, cw, toks)
    size = near.pow(2).mean(-1).sqrt()
    worst = lambda a: ((got - a).pow(2).mean(-1).sqrt() / size).max().item()
    typical = ((got - near).pow(2).mean(-1).sqrt() / size).quantile(0.8).item()
    assert worst(far) > 0.03 and worst(far) > 2 * (worst(near) if name != "routed" else typical), (worst(near), worst(far))


# ---------------------------------------------------------------------------------------------------
# configuration, scheduler, sampling
# ---------------------------------------------------------------------------------------------------
def test_layers_and_their_pools(models):
    cfg, w, path = models("mixed")
    eng = open_engine(path, torch.float32, 256, "cpu")
    m, pools = eng.model, eng.runner.kv.pools
    assert [type(x) for x in m.cfg.mixers] == [RGLRUSpec, LatentSpec, AttnSpec, LatentSpec, RGLRUSpec]
    n, s = eng.runner.kv.num_pages, eng.runner.state_slots + 1
    shapes = [tuple(t.shape) if t is not None else None for pair in pools for t in pair]
    assert shapes == [(s, 96, 3), (s, 96), (n + 1, PAGE, 1, 128 + 16), None, (n, PAGE, 3, 40), (n, PAGE, 3, 24), (n + 1, PAGE, 1, 128 + 32), None, (s, 128, 1), (s, 128)]
    assert pools[0][1].dtype == torch.float32 and m.cfg.has_linear_attn
    assert m.layers[1].mlp.absent and m.layers[1].logits is None and m.layers[0].mlp.experts is not None


@pytest.mark.parametrize("spoil", [lambda c: c["layers"][0].update(type="something"), lambda c: c["layers"][0]["mlp"].update(kind="other"),
                                   lambda c: c["layers"][1]["mixer"]["rot"].update(dims=8)])
def test_unknown_parts_are_refused(spoil):
    cfg = json.loads(json.dumps(CONFIGS["mixed"]))
    spoil(cfg)
    with pytest.raises((NotImplementedError, ValueError)):
        from_hf_dict(cfg)


@pytest.mark.parametrize("where", DEVICES)
def test_greedy_generation(models, where):
    """Engine, scheduler (prompts in portions beside decoded tokens) and sampler: the generated tokens are the argmax of the plain model; the
    same prompts again through used pages and state slots."""
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


@pytest.mark.parametrize("layers", [[(unit(16, 1, 3), moe(2, 1, 16)), (unit(24, 3, 1), None)], [(latent(2, 16, 8, 16, 16, 24), moe(2, 1, 16))], [(attn(2, 1, 16, 16, 8), None)]],
                         ids=["recurrent", "latent", "attention"])
def test_stacks_of_one_kind(tmp_path, layers):
    """Recurrent layers only: no page pools, the scheduler runs on state slots; attention only: no slots, prefixes are reused."""
    cfg = config(layers, width=64, vocab=64)
    w = O.random_weights(cfg, seed=1)
    m = load_model(save(tmp_path / "m", cfg, w), device="cpu", dtype=torch.float32)
    eng = LLMEngine(m, EngineConfig(max_batch=2, max_context=512, max_tokens=1024))
    toks = [(7 * i) % 64 for i in range(150)]
    for _ in range(2):
        out = eng.generate([toks, toks[:3]], GenerationConfig(max_new_tokens=3, ignore_eos=True))
        logits = O.forward(cfg, w, toks + out[0][:-1])[149:]
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
    tiny = random_init(preset("tiny-nasipel"), "cpu", torch.float32)
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
