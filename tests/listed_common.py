"""What the tests of models with listed layers share: devices, checkpoint folders, schedules replayed against a whole-sequence oracle."""
import json

import pytest
import torch

from fastllm_b200.engine.replay import Replay, open_engine
from fastllm_b200.loader import safetensors as st

PAGE = 128
DEVICES = [pytest.param(("cpu", torch.float32), id="cpu"), pytest.param(("cuda", torch.float32), id="gpu32", marks=pytest.mark.gpu),
           pytest.param(("cuda", torch.bfloat16), id="gpu16", marks=pytest.mark.gpu)]


def save(path, cfg, w):
    path.mkdir(exist_ok=True)
    (path / "config.json").write_text(json.dumps(cfg))
    st.save_file(w, path / "model.safetensors")
    return path


@pytest.fixture(autouse=True, scope="module")
def few_threads():
    """The matrices are tiny: more threads than a few only wait for one another."""
    n = torch.get_num_threads()
    torch.set_num_threads(min(n, 4))
    yield
    torch.set_num_threads(n)


def assert_close(got, want, dtype, tol16=0.03, over=0.0):
    """Root mean square of the difference relative to the logits' own, per row; ``over``: the fraction of rows that may miss it in 16
    bits (a head whose output nearly cancels before its norm, an expert chosen by a close call), by a factor of four at most."""
    err = (got.double() - want).pow(2).mean(-1).sqrt() / want.pow(2).mean(-1).sqrt()
    limit = 3e-5 if dtype == torch.float32 else tol16
    bad = (err >= limit).double().mean().item()
    ok = bad <= (over if dtype != torch.float32 else 0.0) and (err.max() < 4 * limit or over > 0.1)
    assert ok, f"relative error {err.max().item():.3g}, {bad:.1%} of the rows over {limit}"


def replay(path, where, reqs, schedule, max_tokens, oracle, over=0.0, tol16=0.03):
    """Run a schedule of (request, count) steps; compares every position's logits with the whole-sequence oracle."""
    device, dtype = where
    eng = open_engine(path, dtype, max_tokens, device)
    rp, at, got = Replay(eng), {}, {r: [] for r in reqs}
    free, slots = eng.pm.num_free(), len(eng.state_free)
    for step in schedule:
        entries = []
        for r, n in step:
            lo = at.get(r, 0)
            entries.append((r, reqs[r][lo:lo + n], list(range(n))))
            at[r] = lo + n
        out = rp.step(entries, [r for r, _ in step if at[r] == len(reqs[r])])
        row = 0
        for r, n in step:
            got[r].append(out[row:row + n])
            row += n
    assert eng.pm.num_free() == free and len(eng.state_free) == slots, "pages or state slots were not given back"
    assert all(at[r] == len(toks) for r, toks in reqs.items())
    assert_close(torch.cat([torch.cat(got[r]) for r in reqs]), torch.cat([oracle(toks) for toks in reqs.values()]), dtype, tol16, over)


def portions(n, sizes):
    out, i = [], 0
    while sum(out) < n:
        out.append(min(sizes[i % len(sizes)], n - sum(out)))
        i += 1
    return out
