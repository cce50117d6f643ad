"""Throughput and kernel times of latent-attention models whose layers are listed one by one, beside the closest other family
(multi-head latent attention with routed experts, DeepSeek-V3 layout) at equal sizes; random weights.

``python bench.py --layers patesun`` prints one JSON line per measurement:
  * ``step``   -- prefill and decode tokens/s of a short stack (one dense layer, three expert layers) through the engine's runner;
  * ``kernel`` -- one operator alone: microseconds, its bytes / FLOPs and the fraction of the measured copy bandwidth or GEMM peak.
Operators are timed with CUDA events behind an L2 flush that also hides the host's launch time; the median of the repeats is kept.
"""
from __future__ import annotations

import json
import os
import statistics

import torch

SIZES = {
    # width, heads, latent rank, window, dense ff, experts, top, expert ff, shared ff
    "2k": dict(width=2048, heads=16, rank=512, window=2048, ff=8192, experts=64, top=6, eff=1024, shared=2048),
    "4k": dict(width=4096, heads=32, rank=512, window=2048, ff=14336, experts=64, top=6, eff=1024, shared=2048),
    "7k": dict(width=7168, heads=128, rank=512, window=4096, ff=18432, experts=64, top=8, eff=2048, shared=2048),
}
HEAD, VOCAB, LAYERS = 128, 32768, 4


def patesun_config(z):
    from ..models.config import from_hf_dict

    mx = {"heads": z["heads"], "dim": HEAD, "vdim": HEAD, "kv_rank": z["rank"], "scale": HEAD ** -0.5, "mask": {"size": z["window"]}}
    moe = {"kind": "moe", "expert": {"ff": z["eff"]}, "router": {"experts": z["experts"], "top": z["top"]}, "shared": {"ff": z["shared"]}}
    return from_hf_dict(dict(architecture="Patesun", vocab=VOCAB, width=z["width"], norm={"eps": 1e-6}, residual_mult=0.4, loop=None,
                             layers=[{"type": "latent_attention", "mixer": mx, "mlp": {"kind": "dense", "ff": z["ff"]} if i == 0 else moe}
                                     for i in range(LAYERS)]))


def mla_config(z):
    from ..models.config import from_hf_dict

    return from_hf_dict(dict(model_type="deepseek_v3", vocab_size=VOCAB, hidden_size=z["width"], num_hidden_layers=LAYERS,
                             num_attention_heads=z["heads"], num_key_value_heads=z["heads"], intermediate_size=z["ff"],
                             moe_intermediate_size=z["eff"], n_routed_experts=z["experts"], num_experts_per_tok=z["top"],
                             n_shared_experts=z["shared"] // z["eff"], first_k_dense_replace=1, n_group=1, topk_group=1,
                             scoring_func="sigmoid", topk_method="noaux_tc", norm_topk_prob=True, kv_lora_rank=z["rank"],
                             qk_nope_head_dim=HEAD, qk_rope_head_dim=64, v_head_dim=HEAD, rms_norm_eps=1e-6, max_position_embeddings=65536))


class Timer:
    def __init__(self, repeats: int = 15):
        self.flush = torch.empty(512 << 20, dtype=torch.uint8, device="cuda")
        self.repeats = repeats

    def us(self, fn) -> float:
        for _ in range(3):
            fn()
        torch.cuda.synchronize()
        out = []
        for _ in range(self.repeats):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            self.flush.fill_(1)
            self.flush.fill_(0)
            a.record()
            fn()
            b.record()
            b.synchronize()
            out.append(a.elapsed_time(b) * 1e3)
        return statistics.median(out)


def peaks() -> tuple[float, float, str]:
    root = os.path.dirname(os.path.dirname(os.path.dirname(os.path.abspath(__file__))))
    try:
        with open(os.path.join(root, "MEASURED_PEAKS.json")) as f:
            d = json.load(f)
        return float(d["hbm_gbs"]), float(d["bf16_tflops"]), "measured"
    except (OSError, KeyError, ValueError):
        return 6650.0, 1590.0, "fallback"


# ---------------------------------------------------------------------------------------------------
# whole steps
# ---------------------------------------------------------------------------------------------------
def bench_steps(family: str, cfg, size: str, cases, emit) -> None:
    from ..engine.runner import EngineConfig, ModelRunner
    from ..models import random_init
    from ..ops import _lib

    model = random_init(cfg, "cuda", torch.bfloat16, seed=0, expert_pool=4)
    gen = torch.Generator().manual_seed(0)
    for batch, ctx in cases:
        pages = (ctx + 64) // 128 + 1
        runner = ModelRunner(model, EngineConfig(max_batch=batch, max_context=pages * 128, prefix_cache=False, graph_batch_sizes=[batch]), num_pages=batch * pages + 1)
        owned = [list(range(b * pages, (b + 1) * pages)) for b in range(batch)]
        toks = torch.randint(0, VOCAB, (ctx,), generator=gen).tolist()
        per = max(1, 8192 // ctx)                       # requests of a prefill step of about 8192 tokens
        n_pre = min(per, batch)

        def prefill(first, count):
            for s in range(0, ctx, 8192):
                runner.prefill([(toks[s:s + 8192], s, owned[b], s + 8192 >= ctx) for b in range(first, first + count)])

        for _ in range(2):
            prefill(0, n_pre)
        torch.cuda.synchronize()
        ms = []
        for _ in range(5):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            prefill(0, n_pre)
            b.record()
            b.synchronize()
            ms.append(a.elapsed_time(b))
        emit(dict(kind="step", family=family, size=size, what="prefill", requests=n_pre, tokens=ctx * n_pre, ms=statistics.median(ms),
                  tokens_per_s=ctx * n_pre / statistics.median(ms) * 1e3))
        for b in range(0, batch, n_pre):
            prefill(b, min(n_pre, batch - b))
        ids = torch.randint(0, VOCAB, (batch,), generator=gen).tolist()
        pos = [ctx] * batch
        for _ in range(4):
            runner.decode(ids, pos, owned)
        slot = runner.slots[batch]
        torch.cuda.synchronize()
        ms = []
        for _ in range(20):
            a, b = torch.cuda.Event(enable_timing=True), torch.cuda.Event(enable_timing=True)
            a.record()
            if slot.graph is not None:
                slot.graph.replay()
            else:
                runner._decode_forward(slot)
            b.record()
            b.synchronize()
            ms.append(a.elapsed_time(b))
        emit(dict(kind="step", family=family, size=size, what="decode", batch=batch, context=ctx, ms=statistics.median(ms),
                  tokens_per_s=batch / statistics.median(ms) * 1e3, launches=runner.launches_per_decode_step, graph=slot.graph is not None))
        _lib.check_device_errors()
        runner.slots.clear()
        del runner, slot
        torch.cuda.empty_cache()
    del model
    torch.cuda.empty_cache()


# ---------------------------------------------------------------------------------------------------
# operators alone: the new one, then the like one of the other family
# ---------------------------------------------------------------------------------------------------
def bench_kernels(z, size: str, emit) -> None:
    from ..models.config import LatentSpec
    from ..models.decoder import ForwardBatch
    from ..ops import attention as A
    from ..ops import basic as B
    from ..ops import latent as LA
    from ..ops import moe as MOE
    from ..ops import stream32 as S

    tm = Timer()
    hbm, tf, src = peaks()
    dev, dt = "cuda", torch.bfloat16
    W, H, R, win = z["width"], z["heads"], z["rank"], z["window"]
    rnd = lambda *s: torch.randn(*s, device=dev, dtype=dt) * 0.05
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=dev)

    def put(name, role, fn, nbytes, flops, **info):
        us = tm.us(fn)
        t_mem, t_mm = nbytes / hbm / 1e3, flops / tf / 1e6           # microseconds at the measured peaks
        emit(dict(kind="kernel", size=size, name=name, role=role, us=round(us, 2), gbytes=nbytes / 1e9, gflop=flops / 1e9,
                  bound="memory" if t_mem > t_mm else "tensor", roofline_frac=round(max(t_mem, t_mm) / us, 4), peak=src, **info))

    # latent decode: windowed latent rows against latent + rotary rows over as many keys
    for batch, ctx in ((64, win), (64, 4 * win)):
        pages = ctx // 128
        lens = i32([ctx] * batch)
        pt = torch.randperm(batch * pages, device=dev).to(torch.int32).view(batch, pages)
        for name, role, dq, w in (("latent_decode", "new", R, win), ("mla_decode", "like", R + 64, 0)):
            pool = rnd(batch * pages + 1, 128, 1, dq)
            q = rnd(batch, H, dq)
            keys = min(ctx, w) if w else ctx
            put(name, role, lambda: A.mla_decode(q, pool, pt, lens, 0.1, lora=R, window=w), batch * (keys * dq * 2 + H * (dq + R) * 2),
                2.0 * batch * H * keys * (dq + R), batch=batch, context=ctx, keys=keys)
            del pool
    # row operators at a prefill-sized batch
    T, top = 8192, z["top"]
    nw, h, y16 = torch.ones(W, device=dev, dtype=dt), torch.randn(T, W, device=dev), rnd(T, W)
    put("rmsnorm32", "new", lambda: S.rmsnorm32(h, nw, 1e-6), T * W * 6, 0)
    put("rmsnorm", "like", lambda: B.rmsnorm(y16, nw, 1e-6), T * W * 4, 0)
    ids, pos = torch.randint(0, VOCAB, (T,), device=dev, dtype=torch.int32), torch.arange(T, device=dev, dtype=torch.int32)
    table, freq = rnd(VOCAB, W), S.sinusoid_inv_freq(W, 10000.0, dev)
    put("embed_pos_norm", "new", lambda: S.embed_pos_norm(ids, pos, table, freq, nw, 1e-6), T * W * 8, 0)
    put("embedding+rmsnorm", "like", lambda: B.rmsnorm(B.embedding(ids, table), nw, 1e-6), T * W * 8, 0)
    rows = T * top
    ys, where, wts = rnd(rows, W), torch.randperm(rows, device=dev).to(torch.int32).view(T, top), torch.full((T, top), 1.0 / top, device=dev)
    put("moe_combine_norm32", "new", lambda: S.moe_combine_norm(ys, where, None, 1.0 / top, y16, h, nw, 0.4, 1e-6), rows * W * 2 + T * W * 12, 0)

    def like_combine():
        out = torch.empty((T, W), device=dev, dtype=dt)
        from ..ops import _lib

        _lib.kernels().fb_moe_combine(B._ptr(ys), B._ptr(where), B._ptr(wts), B._ptr(None), B._ptr(out), T, top, W, 1, B._stream())
        r = out + y16
        return B.rmsnorm(r + y16, nw, 1e-6)
    put("combine+add+add+rmsnorm", "like", like_combine, rows * W * 2 + T * W * 8, 0)
    del ys, where
    # routing plan of the layers of a stack
    class _L:
        pass
    fake = []
    for _ in range(LAYERS - 1):
        l = _L()
        l.route_table = torch.rand((VOCAB, z["experts"]), device=dev).topk(top, dim=1).indices.to(torch.int32).contiguous()
        l.experts = _L()
        l.experts.stacked, l.experts.count = True, z["experts"]
        fake.append(l)
    router = MOE.TableRouter(fake, dev)
    logits, bias = torch.randn(T, z["experts"], device=dev), torch.zeros(z["experts"], device=dev)
    put(f"table plans of {LAYERS - 1} layers", "new", lambda: router.plan(ids), (LAYERS - 1) * T * top * 8, 0)

    def like_plan():
        idx, w_ = MOE.route_topk(logits, bias, top, 1, True)
        c = torch.empty(z["experts"], device=dev, dtype=torch.int32)
        o, t1, p_ = torch.empty_like(c), torch.empty(1, device=dev, dtype=torch.int32), torch.empty((T, top), device=dev, dtype=torch.int32)
        from ..ops import _lib, moe_grouped

        _lib.kernels().fb_moe_plan(B._ptr(idx), T, top, 0, z["experts"], B._ptr(c), B._ptr(o), B._ptr(p_), B._ptr(t1), moe_grouped.PAD, B._stream())
    put("top-k and plan of 1 layer", "like", like_plan, T * top * 8, 0)
    # projections onto the residual
    for M in (64, T):
        x, w, hm, rm = rnd(M, H * HEAD), rnd(W, H * HEAD), torch.randn(M, W, device=dev), rnd(M, W)
        fl = 2.0 * M * W * H * HEAD
        put("gemm_res32", "new", lambda: B.linear_res32(x, w, hm, 0.4), W * H * HEAD * 2 + M * (H * HEAD * 2 + W * 8), fl, rows=M)
        put("gemm_residual", "like", lambda: B.linear(x, w, residual=rm), W * H * HEAD * 2 + M * (H * HEAD * 2 + W * 4), fl, rows=M)
    # prompt chunk: latents -> keys and values -> windowed attention, against the latent-space products of the other family
    spec = LatentSpec(H, HEAD, HEAD, R, HEAD ** -0.5, win)
    lw, _ = LA.build(spec, rnd(H * HEAD, W), rnd(H * HEAD, W), rnd(R, W), torch.ones(R, device=dev, dtype=dt), rnd(H * HEAD, R), rnd(H * HEAD, R))
    for n_req, n in ((1, T), (T // 2048, 2048)):
        pages = n // 128
        cu = [n * b for b in range(n_req + 1)]
        fb = ForwardBatch(ids=ids, positions=pos % n, slots=pos, page_table=torch.arange(n_req * pages, device=dev, dtype=torch.int32).view(n_req, pages),
                          kv_lens=i32([n] * n_req), cu_q=i32(cu), cu_q_host=cu, kv_lens_host=[n] * n_req)
        keys = sum(min(i + 1, win) for i in range(n)) * n_req         # (query, key) pairs
        pool, proj = rnd(n_req * pages + 1, 128, 1, R), rnd(T, lw.latent_col + 64)
        LA.attention(lw, proj, pool, fb)
        grp = fb._latent_plans[next(iter(fb._latent_plans))].groups[0]
        kv = B.linear(S.gather_rows(pool.view(-1, R), grp.key_idx), lw.w_ukv)
        put("latent expand", "new", lambda: B.linear(S.gather_rows(pool.view(-1, R), grp.key_idx), lw.w_ukv), T * (R * 2 + 2 * H * HEAD * 2), 2.0 * T * R * 2 * H * HEAD,
            requests=n_req, tokens=n)
        out = torch.empty((T, H * HEAD), device=dev, dtype=dt)
        put("windowed prefill attention", "new", lambda: LA.window_attention(lw, grp, proj[:, :H * HEAD], proj[:, lw.gate_col:lw.latent_col], kv, out),
            T * H * HEAD * 10, 4.0 * keys * H * HEAD, requests=n_req, tokens=n)
        causal = n * (n + 1) // 2 * n_req
        del kv, out
        if causal * H * 6 / n_req < 40e9:                             # the other family keeps all scores of a request in memory
            q_full, pool2 = rnd(T, H, R + 64), rnd(n_req * pages + 1, 128, 1, R + 64)
            put("mla prefill products", "like", lambda: MOE.mla_paged_attention(q_full, pool2, fb, 0.1, R), T * H * (2 * R + 64) * 2,
                2.0 * causal * H * (2 * R + 64), requests=n_req, tokens=n)
            del q_full, pool2
        torch.cuda.empty_cache()


def run(sizes, steps: bool = True, kernels: bool = True, emit=None) -> None:
    emit = emit or (lambda d: print(json.dumps(d), flush=True))
    for size in sizes:
        z = SIZES[size]
        if kernels:
            bench_kernels(z, size, emit)
        torch.cuda.empty_cache()
        if steps:
            for family, cfg in (("patesun", patesun_config(z)), ("mla", mla_config(z))):
                bench_steps(family, cfg, size, ((1, z["window"]), (64, z["window"] // 2), (64, z["window"])), emit)
