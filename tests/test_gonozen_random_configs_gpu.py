"""Random Gonozen configurations (fixed seeds): widths that are and are not multiples of 8, both mixers in any order and number,
heads and latents of every relation to the tensor-core kernels' sizes, key and value widths equal or not, windows from one
position to longer than the requests or none, rotations of none, some and all of the rotated part, stretched or not, mixtures
of one to twelve experts in one to six groups with and without limits and shared experts, layers without a feed-forward, logits
with and without a bound. Each is replayed whole and as a mixed trace in both element types against the plain restatement, and
some generate through the engine."""
import numpy as np
import pytest

import traces
from test_gonozen_gpu import Ref, against_plain, check_greedy_tokens, lat, lat2, load_plain, model_config, moe, run_trace, write_model, yarn

pytestmark = pytest.mark.gpu

SEEDS = list(range(16))


def random_config(seed):
    rng = np.random.default_rng(6000 + seed)
    pick = lambda xs: xs[int(rng.integers(0, len(xs)))]
    width = pick([50, 64, 90, 104, 128, 160])
    room = [width // 2]                     # coordinates of the stream that the routers may take

    def mlp():
        count = pick([1, 1, 2, 3, 4, 6])
        experts = count * pick([1, 2, 3])
        if rng.random() < 0.25 or experts > room[0]:
            return None
        room[0] -= experts
        keep = int(rng.integers(1, count + 1))
        top = int(rng.integers(1, min(4, keep * (experts // count)) + 1))
        limit = lambda: pick([None, 0.4, 1.0, 2.5])
        return moe(experts, top, pick([8, 21, 64, 72]), limit(), (count, keep) if count > 1 or rng.random() < 0.3 else None,
                   pick([None, (16, limit()), (33, limit()), (64, limit())]))
    layers = []
    for _ in range(int(rng.integers(1, 6))):
        heads, rank, vdim = pick([1, 2, 3, 4, 8]), pick([5, 16, 24, 32, 48, 64, 96, 128, 160]), pick([4, 8, 16, 24, 40, 64])
        stretch = float(rng.uniform(0.6, 1.6))
        if rng.random() < 0.5:
            dim, r = pick([4, 8, 10, 16, 32, 64]), pick([2, 8, 16, 32])
            rot = None if rng.random() < 0.15 else (pick([100.0, 10000.0, 1e6]), pick([r, r, r, 2]))
            if rot and rng.random() < 0.6:
                rot += (yarn(pick([1.5, 2.0, 8.0]), pick([32, 512, 4096]), pick([32.0, 8.0]), pick([1.0, 2.0])),)
            layers.append(lat(heads, dim, r, vdim, rank, rot, round((dim + r) ** -0.5 * stretch, 4), mlp()))
        else:
            dim = pick([4, 7, 8, 16, 32, 64])
            layers.append(lat2(heads, dim, vdim, rank, pick([3, 8, 24, 40, 64]), pick([0, 1, 3, 7, 16, 33, 64, 500]), round(dim ** -0.5 * stretch, 4), mlp()))
    return model_config(int(rng.integers(50, 400)), width, layers, eps=pick([1e-5, 1e-6]), cap=pick([None, 8.0, 20.0, 50.0]))


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
