"""Random Tikizen configurations (fixed seeds): widths that are and are not multiples of 8, the three mixers in any order
and number, head sizes of every relation to the fast kernels' (32, 64, 96, 128 and others), key and value widths equal or
not, one to four key/value heads with one to eight query heads each, chunks from one position to longer than the requests
or none, readers of an earlier layer's keys with masks of their own, rotations of none, some and all of a head's entries,
stretched or not, states of 3 to 136 rows, convolutions of one to five taps, dense and routed feed-forwards with and
without limits and shared experts, and layers without a feed-forward. Each is replayed whole and as a mixed trace in both
element types against the plain restatement, and some generate through the engine."""
import numpy as np
import pytest

import traces
from test_tikizen_gpu import Ref, against_plain, attn, check_greedy_tokens, dense, load_plain, mamba, model_config, moe, ret, run_trace, write_model, yarn

pytestmark = pytest.mark.gpu

SEEDS = list(range(16))


def random_config(seed):
    rng = np.random.default_rng(4000 + seed)
    pick = lambda xs: xs[int(rng.integers(0, len(xs)))]
    width = pick([40, 54, 64, 96, 100, 128, 160])

    def rot(dim, plain_only=False):
        if rng.random() < 0.2:
            return None
        r = (pick([100.0, 10000.0, 1e6]), pick([d for d in (2, 4, 8, 16, 32, 64, dim) if d <= dim and d % 2 == 0]))
        return r if plain_only or rng.random() < 0.4 else r + (yarn(pick([1.5, 2.0, 8.0]), pick([32, 512, 4096]), pick([32.0, 8.0]), pick([1.0, 2.0])),)

    def mlp():
        kind = pick(["none", "dense", "moe", "moe"])
        if kind == "none":
            return None
        if kind == "dense":
            return dense(pick([24, 33, 64, 100]), pick([None, 0.5, 2.0, 7.0]))
        experts = pick([1, 2, 3, 4])
        return moe(experts, int(rng.integers(1, experts + 1)), pick([8, 21, 64, 72]), pick([0, 16, 33, 64]))
    layers = []
    for i in range(int(rng.integers(1, 6))):
        kind = pick(["retention", "attention", "attention", "mamba2"])
        if kind == "retention":
            h, dim = pick([1, 2, 3]), pick([3, 4, 8, 16, 33, 64, 136])
            layers.append(ret(h, dim, pick([4, 8, 24, 40]), rng.uniform(0.8, 1.0, h).round(4).tolist(), rot=rot(dim, True), mlp=mlp()))
        elif kind == "mamba2":
            g = pick([1, 2, 3])
            h, vd = g * pick([1, 2, 3]), pick([3, 8, 16, 32])
            layers.append(mamba(h, vd, pick([3, 8, 16, 33, 64, 130]), g, pick([n for n in (1, 2, 3, h) if (h * vd) % n == 0]), pick([1, 2, 3, 4, 4, 5]), mlp()))
        else:
            sources = [j for j, L in enumerate(layers) if L["type"] == "attention" and "kv_from" not in L["mixer"]]
            chunk = pick([0, 1, 3, 7, 16, 33, 64, 500])
            if sources and rng.random() < 0.5:
                j = pick(sources)
                m = layers[j]["mixer"]
                r = m.get("rot")
                r = None if r is None else (r["base"], r["dims"]) + ((r["scaling"],) if "scaling" in r else ())
                layers.append(attn(m["kv_heads"] * pick([1, 2, 4]), m["kv_heads"], m["dim"], m["vdim"], scale=round(float(rng.uniform(0.1, 0.5)), 3),
                                   chunk=pick([chunk, (m.get("mask") or {}).get("size", 0)]), rot=r, kv_from=j, mlp=mlp()))
            else:
                kv = pick([1, 2, 3, 4])
                dim = pick([6, 8, 16, 20, 32, 48, 64, 72, 96, 128])
                layers.append(attn(kv * pick([1, 2, 4, 8]), kv, dim, pick([dim, dim, dim, 8, 24, 40]),
                                   scale=round(dim ** -0.5 * float(rng.uniform(0.5, 1.5)), 4), chunk=chunk, rot=rot(dim), mlp=mlp()))
    alpha = pick([1.0, 0.7, 1.5, 2.5])
    if any(L["mlp"] and L["mlp"]["kind"] == "moe" for L in layers):
        alpha = max(alpha, 2.0)             # the coordinates that keep the choices of experts apart fade with each sum otherwise
    return model_config(int(rng.integers(50, 400)), width, layers, eps=pick([1e-5, 1e-6]), alpha=alpha)


@pytest.mark.parametrize("seed", SEEDS)
def test_random_configuration(tmp_path, seed):
    config = random_config(seed)
    rng = np.random.default_rng(seed)
    reqs = {f"r{j}": rng.integers(0, config["vocab"], int(n)).tolist() for j, n in enumerate(rng.integers(1, 90, 3))}
    page = [4, 8, 16, 32][seed % 4]
    folder = write_model(tmp_path / "m", config, 77 + seed)
    cfg, w = load_plain(folder)
    ref = {rid: Ref(toks, cfg, w) for rid, toks in reqs.items()}
    assert min(r.margin for r in ref.values()) > 0.05
    for dtype in ("float32", "bfloat16"):
        for fam, make in (("whole", traces.whole), ("mixed", traces.mixed)):
            got = run_trace(folder, dtype, make(reqs), page)
            for rid, toks in reqs.items():
                against_plain(traces.as_matrix(got[rid], len(toks)), ref[rid], dtype, f"seed {seed} {dtype} {fam} {rid}")


@pytest.mark.parametrize("seed", SEEDS[:4])
def test_random_configuration_generates(tmp_path, seed):
    from cellm_b200 import Engine, SamplingParams
    config = random_config(seed)
    folder = write_model(tmp_path / "m", config, 5 + seed)
    cfg, w = load_plain(folder)
    rng = np.random.default_rng(seed)
    prompts = [rng.integers(0, config["vocab"], int(n)).tolist() for n in (3, 40, 17)]
    eng = Engine(folder, dtype="float32", tokens_per_block=8, total_blocks=64, max_num_seqs=2, max_batch_tokens=32, prefill_chunk=16)
    outs = eng.generate(prompts, SamplingParams.greedy(8, stop_eos=False))
    for prompt, out in zip(prompts, outs):
        check_greedy_tokens(cfg, w, prompt, out, "float32")
    s = eng.stats()
    assert s["idle"] and s["free_pages"] == s["total_pages"]
