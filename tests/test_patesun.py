"""Patesun (windowed latent attention, table-routed experts, looped layers, fp32 residual) against its plain statement.

Every case builds a small random model of its own.  The CPU runs use the framework's PyTorch operator definitions (scheduling,
cache, loading and the model itself); the GPU runs the kernels, in float32 and bfloat16.
"""
import json

import pytest
import torch

from . import listed_common as LC
from . import patesun_oracle as O
from .listed_common import DEVICES, PAGE, assert_close, few_threads, portions, save  # noqa: F401
from fastllm_b200.engine import EngineConfig, GenerationConfig, LLMEngine
from fastllm_b200.engine.replay import Replay, open_engine
from fastllm_b200.loader.hf import load_model
from fastllm_b200.models.config import LatentSpec
from fastllm_b200.models.decoder import ForwardBatch
from fastllm_b200.ops import latent as LA
from fastllm_b200.ops import stream32 as S

gpu = pytest.mark.gpu


def mixer(heads, dim, vdim, rank, window, scale=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "scale": scale or dim ** -0.5}
    if window:
        m["mask"] = {"size": window}
    return m


def moe(experts, top, ff, shared):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, "shared": {"ff": shared} if shared else None}


def config(layers, width=160, vocab=304, loop=None, eps=1e-5, mult=0.45):
    return {"architecture": "Patesun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "residual_mult": mult, "loop": loop,
            "layers": [{"type": "latent_attention", "mixer": m, "mlp": f} for m, f in layers]}


CONFIGS = {
    # two windows and head shapes, a loop over two layers, all three kinds of feed-forward
    "mixed": config([(mixer(3, 48, 32, 72, 21), {"kind": "dense", "ff": 208}), (mixer(5, 32, 56, 104, 70), moe(6, 3, 48, 80)),
                     (mixer(2, 64, 16, 40, 21), None), (mixer(4, 40, 40, 136, 150), moe(9, 1, 112, 0))],
                    loop={"start": 1, "stop": 3, "times": 3}),
    # nothing is a multiple of anything the kernels tile
    "odd": config([(mixer(3, 20, 12, 28, 19, scale=0.3), {"kind": "dense", "ff": 75}), (mixer(7, 9, 21, 50, 37), moe(5, 2, 30, 17))],
                  width=148, vocab=331, eps=1e-4, mult=1.0),
    # heads of a served size: several groups of 32 heads, a 512-wide latent, whole tensor-core tiles
    "wide": config([(mixer(36, 128, 128, 512, 200), {"kind": "dense", "ff": 384}), (mixer(16, 192, 128, 256, 333), moe(4, 2, 64, 64))],
                   width=256, vocab=512, mult=0.35),
    # one head, one expert, a window of one token, no loop, and full causal attention
    "ones": config([(mixer(1, 8, 8, 8, 1), moe(1, 1, 8, 8)), (mixer(1, 16, 8, 16, 0), {"kind": "dense", "ff": 8})], width=64, vocab=64, mult=0.7),
}
_CACHE: dict = {}


def weights(name):
    if name not in _CACHE:
        _CACHE[name] = O.random_weights(CONFIGS[name], seed=len(name))
    return _CACHE[name]


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (config, weights, checkpoint folder); the folders are written once."""
    root, out = tmp_path_factory.mktemp("patesun"), {}

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
    LC.replay(models(name)[2], where, reqs, schedule, max_tokens, lambda toks: oracle(name, toks))


# ---------------------------------------------------------------------------------------------------
# the model through cache and batches
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_whole_prompts(models, name, where):
    reqs = {str(n): prompt(name, n) for n in (1, 2, 17, 130, 300)}
    replay(models, name, where, reqs, [[(r, len(t))] for r, t in reqs.items()], 384)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("name", list(CONFIGS))
def test_token_by_token(models, name, where):
    """From the first token on, across two page borders and past every window that is shorter."""
    n = 40 if where[0] == "cpu" else 270
    replay(models, name, where, {"a": prompt(name, n, 1)}, [[("a", 1)]] * n, 384)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("sizes", [(2,), (3, 16, 17), (64, 5), (127, 1, 2), (37, 129, 2, 1)], ids=str)
def test_portions(models, sizes, where):
    n = 150 if where[0] == "cpu" else 300
    for name in ("mixed", "odd", "wide") if where[0] == "cuda" else ("odd",):
        replay(models, name, where, {"a": prompt(name, n, 2)}, [[("a", k)] for k in portions(n, sizes)], 384)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("name", ["mixed", "odd", "wide"])
def test_unequal_requests_and_reused_pages(models, name, where):
    """Up to four live requests: portions beside single tokens, requests that pause, pages used again by later ones."""
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
    # tight pool: "e" and "f" only fit because earlier requests gave their pages back
    replay(models, name, where, reqs, sched, 6 * PAGE)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16], ids=["f32", "bf16"])
def test_long_decoding(models, dtype):
    n = 420
    for name in ("mixed", "wide"):
        replay(models, name, ("cuda", dtype), {"a": prompt(name, n, 9)}, [[("a", 5)]] + [[("a", 1)]] * (n - 5), 512)


# ---------------------------------------------------------------------------------------------------
# window edges: with one layer, a token reaches exactly the rows inside the window behind it
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("window", [1, 2, 31, 64, 100, 128, 129])
def test_window_edge(tmp_path, window, where):
    device, dtype = where
    cfg = config([(mixer(2, 32, 32, 64, window), None)], width=64, vocab=96, mult=2.0)
    w = O.random_weights(cfg, seed=window)
    w["l0.mix.q"] = w["l0.mix.q"] * 3                      # peaked attention: one key among many shows
    path = save(tmp_path / "m", cfg, w)
    n, p = window + 140, 64 if window < 120 else 2
    base = torch.randint(0, 96, (n,), generator=torch.Generator().manual_seed(window)).tolist()
    # the substitute is the token whose latent attracts the edge row's query most
    best = max(range(96), key=lambda t: (O.forward(cfg, w, base[:p] + [t] + base[p + 1:p + window])[-1] - O.forward(cfg, w, base[:p + window])[-1]).abs().max().item())
    other = base[:p] + [best] + base[p + 1:]
    eng = open_engine(path, dtype, 512, device)
    for cut in ([n], [p + window // 2 + 1, n - p - window // 2 - 1], [p + 1] + [1] * (n - p - 1) if device == "cuda" or window < 40 else [n]):
        outs = []
        for seq in (base, other):
            rp, at, rows = Replay(eng), 0, []
            for k in cut:
                rows.append(rp.step([("r", seq[at:at + k], list(range(k)))], ["r"] if at + k == n else []))
                at += k
            outs.append(torch.cat(rows))
        diff = (outs[0] - outs[1]).abs().amax(-1)
        noise = 1e-4 if dtype == torch.float32 else 0.02
        assert diff[p + window - 1] > 5 * noise, "the last row inside the window does not see the token"
        assert diff[:p].max() < noise and diff[p + window:].max() < noise, "a row outside the window sees the token"


# ---------------------------------------------------------------------------------------------------
# mechanisms alone
# ---------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("width", [64, 148, 75])
def test_embedding_positions_and_norm(width, where):
    device, dtype = where
    g = torch.Generator().manual_seed(width)
    table = torch.randn(50, width, generator=g).to(torch.bfloat16)
    nw = torch.randn(width, generator=g).to(torch.bfloat16)
    ids = torch.randint(0, 50, (9,), generator=g)
    pos = torch.tensor([0, 1, 2, 3, 127, 128, 4095, 70001, 999_999])
    h, y = S.embed_pos_norm(ids.int().to(device), pos.int().to(device), table.to(device, dtype), S.sinusoid_inv_freq(width, 10000.0, device),
                            nw.to(device, dtype), 1e-5)
    want = table[ids].double() + O.sinusoid(pos, width)
    assert (h.cpu().double() - want).abs().max() < 1e-6 * 8
    assert (y.cpu().double() - O.rms_norm(want, nw.double(), 1e-5)).abs().max() < (2e-5 if dtype == torch.float32 else 0.06)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("width", [8, 76, 201, 512])
def test_norms(width, where):
    """fp32 rows, and latent rows into cache slots with padded entries and rows that are not cached."""
    device, dtype = where
    g = torch.Generator().manual_seed(width)
    x = torch.randn(7, width, generator=g) * 3 + 0.5
    w = (1 + 0.3 * torch.randn(width, generator=g)).to(torch.bfloat16)
    got = S.rmsnorm32(x.to(device), w.to(device, dtype), 1e-3).cpu().double()
    want = O.rms_norm(x.double(), w.double(), 1e-3)
    assert (got - want).abs().max() < (1e-5 if dtype == torch.float32 else 0.05)
    ld = (width + 7) // 8 * 8
    pool = torch.full((3, PAGE, 1, ld), 7.0, device=device, dtype=dtype)
    slots = torch.tensor([5, -1, 130, 0, 127, 128, -1], dtype=torch.int32)
    xs = x.to(device, dtype)
    S.latent_post(xs, 0, w.to(device, dtype), width, slots.to(device), pool, 1e-3)
    flat = pool.view(-1, ld).cpu().double()
    want = O.rms_norm(xs.cpu().double(), w.double(), 1e-3)
    for t, s in enumerate(slots.tolist()):
        if s >= 0:
            assert (flat[s, :width] - want[t]).abs().max() < (1e-5 if dtype == torch.float32 else 0.05) and flat[s, width:].abs().sum() == 0
    assert (flat[1] == 7).all() and (flat[256] == 7).all()


def _latent_case(spec, lens, news, device, dtype, seed=0, strong=()):
    """Cached latents of requests with ``lens`` tokens, of which the last ``news`` are this batch's.  ``strong``: (request, query
    index, key index, score): that query meets that key with this score in every head."""
    g = torch.Generator().manual_seed(seed)
    H, D, V, R = spec["heads"], spec["dim"], spec["vdim"], spec["kv_rank"]
    r16 = lambda *s: torch.randn(*s, generator=g).to(torch.bfloat16)
    uk, uv = r16(H * D, R) * R ** -0.5, r16(H * V, R) * R ** -0.5
    c = [r16(n, R) for n in lens]
    q, gate = [r16(n, H * D) for n in news], [r16(n, H * V) for n in news]
    for b, i, j, score in strong:
        k = O.linear(uk, c[b][j:j + 1].double()).reshape(H, D)
        q[b][i] = (k * (score / spec["scale"] / k.pow(2).sum(-1, keepdim=True))).reshape(-1).to(torch.bfloat16)
    want = torch.cat([O.latent_core(q[b].double(), c[b].double(), uk.double(), uv.double(), gate[b].double(), spec) for b in range(len(lens))])
    sp = LatentSpec(H, D, V, R, spec["scale"], (spec.get("mask") or {}).get("size") or 0)
    zero = torch.zeros(H * D, 16)
    to = lambda t: t.to(device, dtype)
    lw, _, _ = LA.build(sp, to(zero), to(torch.zeros(H * V, 16)), to(torch.zeros(R, 16)), to(torch.ones(R)), to(uk), to(uv))
    # pages are handed out in a shuffled order; a page of every request starts dirty
    npg = [(n + PAGE - 1) // PAGE for n in lens]
    order = torch.randperm(sum(npg), generator=g).tolist()
    pool = torch.full((sum(npg) + 1, PAGE, 1, lw.ld), 3.0, dtype=dtype)
    table = torch.zeros((len(lens), max(npg)), dtype=torch.int32)
    for b, n in enumerate(lens):
        for i in range(npg[b]):
            table[b, i] = pg = order.pop()
            rows = c[b][i * PAGE:(i + 1) * PAGE]
            pool[pg, :len(rows), 0] = 0
            pool[pg, :len(rows), 0, :R] = rows.to(dtype)
    T = sum(news)
    proj = torch.zeros((T, (lw.latent_col + 31) // 32 * 32), dtype=dtype)
    proj[:, :H * lw.dim].view(T, H, lw.dim)[..., :D] = torch.cat(q).to(dtype).view(T, H, D)
    proj[:, lw.gate_col:lw.latent_col].view(T, H, lw.vdim)[..., :V] = torch.cat(gate).to(dtype).view(T, H, V)
    cu = [0]
    for n in news:
        cu.append(cu[-1] + n)
    pos = torch.cat([torch.arange(n - k, n) for n, k in zip(lens, news)]).int()
    mv = lambda t: t.to(device)
    fb = ForwardBatch(ids=mv(pos), positions=mv(pos), slots=mv(pos), page_table=mv(table), kv_lens=mv(torch.tensor(lens, dtype=torch.int32)),
                      cu_q=mv(torch.tensor(cu, dtype=torch.int32)), cu_q_host=cu, is_decode=all(n == 1 for n in news), kv_lens_host=lens)
    got = LA.attention(lw, mv(proj), mv(pool), fb).cpu().double().view(T, H, lw.vdim)[..., :V].reshape(T, H * V)
    return got, want


def _check_latent(spec, lens, news, where, **kw):
    device, dtype = where
    got, want = _latent_case(spec, lens, news, device, dtype, **kw)
    err = (got - want).abs().amax(-1)
    tol = 2e-5 if dtype == torch.float32 else 0.05
    assert err.max() < tol, (err.argmax().item(), err.max().item())


SPECS = [mixer(4, 32, 24, 64, 41), mixer(3, 24, 8, 20, 129), mixer(40, 128, 128, 512, 1000), mixer(8, 96, 112, 200, 128), mixer(17, 192, 128, 448, 64),
         mixer(2, 64, 200, 320, 77), mixer(2, 16, 16, 640, 50), mixer(5, 64, 64, 128, 0)]


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("spec", SPECS, ids=lambda s: "-".join(str(s[k]) for k in ("heads", "dim", "vdim", "kv_rank")) + f"-w{(s.get('mask') or {}).get('size', 0)}")
def test_latent_attention(spec, where):
    """Decoded tokens, prompt chunks (one and several 128- and 256-row blocks), short portions, and all of them in one batch."""
    _check_latent(spec, [1, 2, 40, 41, 128, 129, 300, 1100], [1] * 8, where)
    _check_latent(spec, [700], [700], where, seed=1)
    _check_latent(spec, [17, 300, 1100, 129, 600], [17, 257, 130, 128, 18], where, seed=2)
    _check_latent(spec, [500, 260, 90, 1030, 33], [1, 200, 2, 300, 16], where, seed=3)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("spec", [mixer(4, 32, 24, 64, 41), mixer(9, 128, 128, 256, 130), mixer(2, 24, 40, 104, 257)], ids=["w41", "w130", "w257"])
def test_far_keys_stand_out(spec, where):
    """One key carries nearly all of a query's weight: at the window's first key, one before it (unseen), at page borders and far
    back, for decoded rows and for rows of a chunk."""
    W = spec["mask"]["size"]
    n = 3 * W + 300
    for news in (1, 2, 16, 17, 300) if where[0] == "cuda" else (1, 300):
        for i in sorted({0, news // 2, news - 1}):
            at = n - news + i                                       # position of the query
            for j in {at, at - W + 1, at - W, at - W // 2, (at // PAGE) * PAGE, (at // PAGE) * PAGE - 1, at - W - 100}:
                if 0 <= j <= at:
                    _check_latent(spec, [n, 200], [news, 1], where, seed=j, strong=[(0, i, j, 14.0)])


@pytest.mark.parametrize("where", DEVICES)
def test_many_absorbed_rows(where):
    """More rows than one call of the latent decode kernel takes."""
    n = 70 if where[0] == "cuda" else 3
    _check_latent(mixer(2, 32, 32, 64, 50), [200 + b for b in range(n)], [16] * n, where)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("shape", [(6, 3, 48, 80, 160), (9, 1, 112, 0, 256), (64, 6, 64, 128, 384), (1, 1, 8, 8, 72)], ids=str)
@pytest.mark.parametrize("rows", [1, 7, 300])
def test_table_experts(tmp_path, shape, rows, where):
    """Routing plan, grouped experts, shared expert, combine onto the residual and the next norm (one layer of a model)."""
    device, dtype = where
    E, top, ff, sh, width = shape
    cfg = config([(mixer(1, 8, 8, 8, 4), moe(E, top, ff, sh))], width=width, vocab=112)
    w = O.random_weights(cfg, seed=E)
    m = load_model(save(tmp_path / "m", cfg, w), device=device, dtype=dtype)
    g = torch.Generator().manual_seed(rows)
    ids = torch.randint(0, 112, (rows,), generator=g)
    h0, x = torch.randn(rows, width, generator=g), torch.randn(rows, width, generator=g).to(torch.bfloat16)
    h = h0.clone().to(device)
    fb = ForwardBatch(ids=ids.int().to(device), positions=None, slots=None, page_table=None, kv_lens=None, cu_q=None)
    h, y = m._mlp(m.layers[0].mlp, x.to(device, dtype), h, 0, m.final_norm, None, fb)
    wd = {k: v.double() if v.is_floating_point() else v for k, v in w.items()}
    want = h0.double() + cfg["residual_mult"] * O.table_moe(x.double(), ids, wd, "l0.mlp.", cfg["layers"][0]["mlp"])
    tol = 3e-5 if dtype == torch.float32 else 0.01 * (want - h0).abs().max()
    assert (h.cpu().double() - want).abs().max() < tol
    assert (y.cpu().double() - O.rms_norm(want, wd["final.norm"], 1e-5)).abs().max() < (1e-4 if dtype == torch.float32 else 0.1)


@pytest.mark.parametrize("where", DEVICES)
@pytest.mark.parametrize("rows,ff,width", [(1, 208, 160), (5, 75, 148), (300, 512, 256), (700, 96, 320)])
def test_relu2_feed_forward(tmp_path, rows, ff, width, where):
    device, dtype = where
    cfg = config([(mixer(1, 8, 8, 8, 4), {"kind": "dense", "ff": ff})], width=width, vocab=64, mult=0.6)
    w = O.random_weights(cfg, seed=ff)
    m = load_model(save(tmp_path / "m", cfg, w), device=device, dtype=dtype)
    g = torch.Generator().manual_seed(rows)
    h0, x = torch.randn(rows, width, generator=g), torch.randn(rows, width, generator=g).to(torch.bfloat16)
    h, _ = m._mlp(m.layers[0].mlp, x.to(device, dtype), h0.clone().to(device), 0, m.final_norm, None, None)
    want = h0.double() + 0.6 * O.relu2_ff(x.double(), {k: v.double() for k, v in w.items() if v.is_floating_point()}, "l0.mlp.")
    assert (h.cpu().double() - want).abs().max() < (3e-5 if dtype == torch.float32 else 0.05)


# ---------------------------------------------------------------------------------------------------
# configuration, scheduler, sampling
# ---------------------------------------------------------------------------------------------------
def test_layer_runs_have_their_own_caches(models):
    cfg, _, path = models("mixed")
    eng = open_engine(path, torch.float32, 256, "cpu")
    m = eng.model
    assert m.cfg.layer_runs == [0, 1, 2, 1, 2, 1, 2, 3] == O.layer_order(cfg)
    assert m.layers[1] is m.layers[3] is m.layers[5] and m.layers[2] is m.layers[6]
    pools = [p[0] for p in eng.runner.kv.pools]
    assert len({p.data_ptr() for p in pools}) == 8
    assert [p.shape[-1] for p in pools] == [72, 104, 40, 104, 40, 104, 40, 136]


def test_unknown_parts_are_refused():
    from fastllm_b200.models.config import from_hf_dict

    cfg = json.loads(json.dumps(CONFIGS["ones"]))
    cfg["layers"][0]["type"] = "something_else"
    with pytest.raises(NotImplementedError):
        from_hf_dict(cfg)


@pytest.mark.parametrize("where", DEVICES)
def test_greedy_generation(models, where):
    """The engine's own scheduler: chunked prompts beside decoding requests, eviction-free pool, arg-max of the plain model."""
    device, dtype = where
    name, n_new = "mixed", 6
    cfg, w, path = models(name)
    m = load_model(path, device=device, dtype=dtype)
    eng = LLMEngine(m, EngineConfig(max_batch=4, max_context=512, chunked_prefill_size=50), num_pages=20)
    prompts = [prompt(name, k, 20) for k in (1, 60, 133)]
    outs = eng.generate(prompts, GenerationConfig(max_new_tokens=n_new, ignore_eos=True))
    for p, out in zip(prompts, outs):
        assert len(out) == n_new
        logits = O.forward(cfg, w, p + out[:-1])[len(p) - 1:]
        for k, t in enumerate(out):                                 # a near tie may fall either way in 16 bits
            gap = (logits[k].max() - logits[k][t]).item()
            assert gap < (1e-4 if dtype == torch.float32 else 0.05), (k, gap)
    # the same prompts again hit the prefix cache's whole pages and give the same tokens
    again = eng.generate(prompts, GenerationConfig(max_new_tokens=n_new, ignore_eos=True))
    assert again == outs or dtype != torch.float32
    assert eng.pm.stats()["hits"] > 0


@gpu
@pytest.mark.parametrize("wdtype", ["int8", "fp8", "int4g128"])
def test_quantised_weights(models, wdtype):
    """Run-time weight formats: the same model with coarser weights, decoding through captured graphs."""
    cfg, w, path = models("wide")
    m = load_model(path, device="cuda", wdtype=wdtype)
    rp = Replay(LLMEngine(m, EngineConfig(max_batch=4, max_context=256, prefix_cache=False), num_pages=4))
    toks = prompt("wide", 150, 40)
    got = torch.cat([rp.step([("a", toks[:140], list(range(140)))])] + [rp.step([("a", toks[i:i + 1], [0])]) for i in range(140, 150)])
    assert_close(got, oracle("wide", toks), torch.bfloat16, 0.1 if wdtype != "int4g128" else 0.4)


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
    assert len(out) == 4 and all((want[k].max() - want[k][t]) < 0.05 for k, t in enumerate(out))
    tiny = random_init(preset("tiny-patesun"), "cpu", torch.float32)
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
