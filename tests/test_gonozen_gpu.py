"""The Gonozen design against its plain restatement (tests/plain_gonozen.py): the kernels of each mechanism alone, whole
models in every cutting of the requests, pages and slots that are used again, keys at the edge of a window and far away,
sinks, gates, the first tokens of a sequence, long decoding through windows and pages, sizes that differ in everything, and
greedy generation through the engine and its command lines."""
import json
import math
import os
import re
import subprocess
import sys
from dataclasses import replace

import numpy as np
import pytest
import torch

import plain_gonozen as plain
import traces
from tolerances import K, K_SELF, check_close

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def yarn(factor, original, fast=32.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def lat(heads, dim, rot_dim, vdim, rank, rot=None, scale=None, mlp=None):
    """rot: (base, dims) or (base, dims, scaling)."""
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": rank, "scale": scale if scale is not None else (dim + rot_dim) ** -0.5}
    if rot is not None:
        m["rot"] = {"base": rot[0], "dims": rot[1], **({"scaling": rot[2]} if len(rot) > 2 else {})}
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def lat2(heads, dim, vdim, rank, q_rank, window=0, scale=None, mlp=None):
    m = {"heads": heads, "dim": dim, "vdim": vdim, "kv_rank": rank, "q_rank": q_rank, "scale": scale if scale is not None else dim ** -0.5}
    if window:
        m["mask"] = {"size": window}
    return {"type": "latent_attention_2", "mixer": m, "mlp": mlp}


def moe(experts, top, ff, limit=None, groups=None, shared=None):
    """groups: (count, keep); shared: (ff, limit)."""
    e = lambda f, l: {"ff": f} if l is None else {"ff": f, "limit": l}
    d = {"kind": "moe", "expert": e(ff, limit), "router": {"experts": experts, "top": top}}
    if groups:
        d["router"]["groups"] = {"count": groups[0], "keep": groups[1]}
    if shared:
        d["shared"] = e(*shared)
    return d


def model_config(vocab, width, layers, eps=1e-5, cap=25.0):
    return {"architecture": "Gonozen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "layers": layers, **({"logit_softcap": cap} if cap else {})}


# A: both mixers; key, value and latent widths that differ every way; windows shorter and longer than pages; stretched and
# plain frequencies; one and several kept groups, with and without a shared expert; a layer without a feed-forward
CONFIG_A = model_config(300, 96, [
    lat2(3, 16, 24, 40, 28, window=21, mlp=moe(8, 2, 40, 0.8, (4, 2), (56, 1.3))),
    lat(4, 16, 8, 12, 32, rot=(5000.0, 8, yarn(4.0, 512)), mlp=moe(6, 3, 24, 1.0, (3, 2))),
    lat2(2, 24, 8, 24, 20, window=64),
    lat(2, 8, 16, 16, 48, rot=(300.0, 16), mlp=moe(4, 1, 33, 2.0, (2, 1), (20, 0.5))),
], cap=14.0)
# B: sizes that are multiples of nothing; windows of one position and none; one head, one expert of one, no groups, no limits,
# no rotation, a rotation of part of the rotated values, logits as they are
CONFIG_B = model_config(211, 54, [
    lat2(3, 5, 7, 11, 9, window=1, mlp=moe(1, 1, 9, 1.1)),
    lat(2, 6, 4, 10, 13, rot=(77.0, 2)),
    lat2(1, 10, 6, 17, 3, window=50, scale=0.9, mlp=moe(6, 2, 13, None, (6, 4), (7, None))),
    lat(3, 10, 6, 5, 7, mlp=moe(5, 5, 21, 0.4)),
    lat2(2, 7, 9, 21, 30),
], eps=1e-6, cap=None)
# C: widths that the tensor-core kernels take (latents whose values split over one, two, five and seven groups of warps)
CONFIG_C = model_config(512, 256, [
    lat(8, 64, 32, 64, 128, rot=(20000.0, 32, yarn(2.0, 1024)), mlp=moe(16, 4, 64, 1.5, (4, 3), (128, 2.5))),
    lat2(4, 32, 64, 64, 96, window=100, mlp=moe(32, 6, 96, 0.7, (8, 4), (64, 0.9))),
    lat(16, 32, 32, 32, 224, rot=(10000.0, 32), mlp=moe(16, 2, 128, 1.0, (2, 1))),
    lat2(5, 48, 80, 80, 64, window=33, mlp=moe(9, 2, 72, 1.2, (3, 2), (40, 1.0))),
], cap=30.0)
# D: long rows (a latent of 512), two heads, a width the tensor-core products do not take
CONFIG_D = model_config(157, 100, [
    lat(2, 128, 64, 128, 512, rot=(10000.0, 64, yarn(8.0, 64, 8.0, 2.0)), mlp=moe(4, 4, 30, 0.9, None, (50, 1.4))),
    lat2(2, 64, 64, 256, 128, window=40, mlp=moe(3, 2, 20, 1.7, (3, 2))),
    lat(1, 20, 12, 140, 24, rot=(50.0, 12)),
], cap=9.0)
CONFIGS = {"a": CONFIG_A, "b": CONFIG_B, "c": CONFIG_C, "d": CONFIG_D}
LENGTHS = {"a": [1, 9, 40, 64, 131, 77, 2], "b": [3, 55, 150, 18, 97], "c": [200, 1, 65, 129, 30, 230], "d": [70, 2, 33, 140, 17]}
PAGE = {"a": 8, "b": 16, "c": 16, "d": 4}


def steer_routers(tensors, config, seed):
    """Gives every mixture `experts` coordinates of the stream: each token's embedding row is largest in the chosen ones, smaller
    in one other of each kept group, negative elsewhere; the norms behind the sublayers let little of their results through
    there, and the router reads these coordinates with a large weight beside its random ones. The choices of groups and of
    experts then differ from token to token but none is close, so that a 16-bit rounding changes none."""
    rng = np.random.default_rng(seed)
    V, at = config["vocab"], 0
    mixtures = [(i, L["mlp"]["router"]) for i, L in enumerate(config["layers"]) if L.get("mlp")]
    total = sum(r["experts"] for _, r in mixtures)
    assert total <= config["width"] // 2, "the routers' coordinates leave the stream too little room"
    for name, t in tensors.items():
        if total and name.endswith(("norm1b", "norm2b")):
            t[:total] *= 0.02
    for i, r in mixtures:
        E, top = r["experts"], r["top"]
        n, keep = (r["groups"]["count"], r["groups"]["keep"]) if r.get("groups") else (1, 1)
        size = E // n
        code = np.full((V, E), -1.0)
        for t in range(V):
            kept = rng.permutation(n)[:keep]
            members = rng.permutation(np.concatenate([np.arange(g * size, (g + 1) * size) for g in kept]))
            chosen = members[:top]
            code[t, chosen] = 1.0
            for g in kept:                              # a kept group of which nothing is chosen still ranks above those left out
                inside = np.arange(g * size, (g + 1) * size)
                if not np.isin(inside, chosen).any():
                    code[t, inside[0]] = 0.0
        std = float(tensors["embed"].float()[:, total:].std())
        code = code * 2.5 * std + rng.uniform(-0.2, 0.2, (V, E)) * std
        tensors["embed"][:, at:at + E] = torch.tensor(code).to(tensors["embed"].dtype)
        router = tensors[f"l{i}.mlp.router"].float() * 0.1
        router[:, at:at + E] += 6.0 * torch.eye(E)
        tensors[f"l{i}.mlp.router"] = router.to(tensors[f"l{i}.mlp.router"].dtype)
        at += E


def write_model(folder, config, seed, dtype="bfloat16", init=None):
    from cellm_b200.weights import InitSpec, write_random_model
    from cellm_b200.weights.safetensors_io import SafetensorsFile, save_file
    # matrices whose products of a normed vector have a size near one: scores neither flat nor so sharp that they pass every rounding on
    init = init or InitSpec(linear_std=1.2 * config["width"] ** -0.5, embedding_std=0.8, bias_std=0.3, norm_jitter=0.2)
    folder = write_random_model(str(folder), config, seed, dtype, init)
    path = os.path.join(folder, "model.safetensors")
    sf = SafetensorsFile(path)
    tensors = {n: sf.tensor(n).clone() for n in sf.names()}
    sf.close()
    steer_routers(tensors, config, seed)
    save_file(tensors, path, {"format": "pt"})
    return folder


def load_plain(folder):
    from cellm_b200.weights.safetensors_io import SafetensorsFile
    with open(os.path.join(folder, "config.json")) as f:
        cfg = json.load(f)
    sf = SafetensorsFile(os.path.join(folder, "model.safetensors"))
    return cfg, {n: sf.tensor(n).to(torch.float64) for n in sf.names()}


def run_trace(folder, dtype, steps, page, use_graphs=True, max_tokens=None):
    from cellm_b200.replay import Replayer
    rp = Replayer(folder, dtype, max_tokens or traces.max_live_tokens(steps), page, 4, use_graphs=use_graphs)
    outs = [rp.step(s["entries"], s["end"]) for s in steps]
    assert rp.cache.live == 0
    assert all(rp.cache.free_pages(g) == rp.cache.group_pages[g] for g in range(len(rp.cache.group_pages)))
    return traces.collect(steps, outs)


class Ref(np.ndarray):
    """A request's plain logits [T, vocab] and, as `.spread` [T], how far `runs` runs whose every product and norm was
    disturbed by a 16-bit rounding's worth (1 + 2^-9 u, u uniform in [-1, 1)) moved each row; `.margin`: the smallest
    distance (of router sums) by which a choice of groups or experts was made."""
    def __new__(cls, toks, cfg, w, runs=2):
        margins = []
        exact = plain.forward(toks, cfg, w, margins=margins)
        self = np.asarray(exact.numpy()).view(cls)
        spread = torch.zeros(len(toks), dtype=torch.float64)
        for seed in range(runs):
            with plain.disturbed(2.0 ** -9, seed):
                spread = torch.maximum(spread, (plain.forward(toks, cfg, w) - exact).abs().amax(dim=1))
        self.spread = spread.numpy()
        self.margin = min((float(m.min()) for m in margins), default=math.inf)
        return self


@pytest.fixture(scope="module")
def models(tmp_path_factory):
    """name -> (folder, requests, plain logits)."""
    d = tmp_path_factory.mktemp("gz")
    out = {}
    for i, (name, config) in enumerate(CONFIGS.items()):
        rng = np.random.default_rng(171 + i)
        reqs = {f"r{j}": rng.integers(0, config["vocab"], n).tolist() for j, n in enumerate(LENGTHS[name])}
        folder = write_model(d / name, config, 127 + i)
        cfg, w = load_plain(folder)
        out[name] = (folder, reqs, {rid: Ref(toks, cfg, w) for rid, toks in reqs.items()})
    return out


# Against the plain restatement in 64-bit: 32-bit sums reordered through up to five layers whose every result is divided by its
# root mean square, 1e-5 of the logits' size; bfloat16 keeps the engine's bound, except for rows that rounding alone moves further.
KP = {"float32": 1e-5, "bfloat16": K["bfloat16"]}


def against_plain(got, ref, dtype, what, k32=None):
    """32-bit: one bound for all rows (`k32`: another than the usual one). bfloat16: a row that rounding alone moves further
    than the engine's bound (measured on the plain model) is held to four times that movement instead."""
    if dtype == "float32":
        return check_close(got, ref, dtype, what, k=k32 or KP[dtype])
    got, exact = np.asarray(got, dtype=np.float64), np.asarray(ref, dtype=np.float64)
    assert got.shape == exact.shape and np.isfinite(got).all(), what
    tol = np.maximum(KP[dtype] * (1.0 + np.abs(exact).max()), 4.0 * ref.spread)
    err = np.abs(got - exact).max(axis=1)
    bad = np.nonzero(err > tol)[0]
    assert bad.size == 0, f"{what}: row {bad[0]} is off by {err[bad[0]]:.3e} > {tol[bad[0]]:.3e} ({bad.size} rows of {len(err)})"


FAMILIES = {"whole": traces.whole, "tail": traces.tail_one_by_one, "portions": traces.portions, "mixed": traces.mixed}


# ---------------------------------------------------------------------------------------------- whole models
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", list(CONFIGS))
def test_every_cutting_matches_plain(models, name, dtype):
    folder, reqs, ref = models[name]
    assert min(r.margin for r in ref.values()) > 0.1            # no choice of experts is close
    results = {}
    for fam, make in FAMILIES.items():
        got = results[fam] = run_trace(folder, dtype, make(reqs), PAGE[name])
        for rid, toks in reqs.items():
            against_plain(traces.as_matrix(got[rid], len(toks)), ref[rid], dtype, f"{name} {dtype} {fam} {rid}")
    for fam in ("tail", "portions", "mixed"):
        for rid, toks in reqs.items():
            check_close(traces.as_matrix(results[fam][rid], len(toks)), traces.as_matrix(results["whole"][rid], len(toks)),
                        dtype, f"{name} {dtype} {fam} vs whole {rid}", k=K_SELF[dtype] if dtype == "bfloat16" else 4e-6)
    got = run_trace(folder, dtype, traces.mixed(reqs), PAGE[name], use_graphs=False)
    for rid, toks in reqs.items():
        check_close(traces.as_matrix(got[rid], len(toks)), traces.as_matrix(results["mixed"][rid], len(toks)), dtype,
                    f"{name} {dtype} mixed: kernel by kernel vs graphs {rid}", k=K_SELF[dtype])


@pytest.mark.parametrize("name", ["a", "b"])
def test_the_model_cut_after_every_layer(models, name):
    """The first n layers of a model for every n, through the last norm and the output, against the plain ones; and the block
    run part by part through its own forward() gives the executor's stream."""
    from cellm_b200.models import load_model
    from cellm_b200.parts import block as B
    from cellm_b200.replay import Replayer
    folder, reqs, _ = models[name]
    cfg, w = load_plain(folder)
    toks = reqs["r3"]
    outs = {}
    for by_parts in (False, True):
        emit = B.SandwichNormBlock.emit
        if by_parts:
            B.SandwichNormBlock.emit = B.Block.emit
        try:
            loaded = load_model(folder, "float32")
            run = loaded[2].forward
            for n in range(len(cfg["layers"]) + 1):
                loaded[2].forward = lambda ctx, bindings, rows, max_layers=None: run(ctx, bindings, rows, n)
                rp = Replayer(loaded, "float32", 64, 8, 4, use_graphs=False)
                outs[by_parts, n] = rp.step([{"id": "x", "tokens": toks, "want": list(range(len(toks)))}], ["x"])
                ref = plain.forward(toks, {**cfg, "layers": cfg["layers"][:n]}, w).numpy()
                check_close(outs[by_parts, n], ref, "float32", f"the first {n} layers", k=KP["float32"])
        finally:
            B.SandwichNormBlock.emit = emit
    for n in range(len(cfg["layers"]) + 1):
        check_close(outs[True, n], outs[False, n], "float32", f"by parts, {n} layers", k=K_SELF["float32"])


def test_mixed_trace_reuses_pages_and_slots(models):
    folder, reqs, _ = models["a"]
    steps = traces.mixed(reqs)
    assert len(reqs) > 4                                     # more requests than may live at once
    assert traces.max_live_tokens(steps) < sum(-(-len(t) // 64) * 64 for t in reqs.values())


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["b", "c"])
def test_portions_of_two_and_odd_sizes(models, name, dtype):
    folder, reqs, ref = models[name]
    for sizes in ((2,), (3, 2, 5), (17, 2, 2, 31), (1, 1, 2)):
        got = run_trace(folder, dtype, traces.portions(reqs, sizes), PAGE[name])
        for rid, toks in reqs.items():
            against_plain(traces.as_matrix(got[rid], len(toks)), ref[rid], dtype, f"{name} {dtype} portions {sizes} {rid}")


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", ["a", "c"])
def test_long_decoding_through_windows_and_pages(models, name, dtype):
    """Most of the sequence decoded token by token: windows move over decoded tokens, and the pages behind them are given back
    while the request lives."""
    folder, reqs, ref = models[name]
    some = {rid: reqs[rid] for rid in (("r4", "r5") if name == "a" else ("r0", "r5"))}
    got = run_trace(folder, dtype, traces.tail_one_by_one(some, tail=190), 8)
    for rid, toks in some.items():
        against_plain(traces.as_matrix(got[rid], len(toks)), ref[rid], dtype, f"{name} {dtype} long tail {rid}")


def test_a_windowed_request_holds_its_window_only(tmp_path):
    """A request longer than the pools of its layers runs through, and the logits are the plain model's."""
    from cellm_b200.replay import Replayer
    config = model_config(120, 48, [lat2(2, 8, 6, 12, 10, window=20, mlp=moe(4, 2, 12, 1.0, (2, 1))), lat2(3, 4, 8, 12, 5, window=20), lat2(1, 9, 5, 12, 4, window=9)])
    folder = write_model(tmp_path / "w", config, 3)
    cfg, w = load_plain(folder)
    toks = np.random.default_rng(0).integers(0, 120, 210).tolist()
    ref = plain.forward(toks, cfg, w).numpy()
    rp = Replayer(folder, "float32", 64, 8, 4)               # 8 pages of 8 tokens a group: 64 rows for 210 tokens
    rows = []
    for i in range(0, len(toks), 5):
        part = toks[i:i + 5]
        rows.append(rp.step([{"id": "x", "tokens": part, "want": list(range(len(part)))}], []))
        n = i + len(part)
        for g, need in enumerate(rp.cache.paged_keys):
            table = rp.cache.block_table(0, g, np.full((64,), -1, dtype=np.int32))
            assert [p >= 0 for p in table] == [(b + 1) * 8 > n - need.window + 1 for b in range(len(table))], (n, g)
    assert sorted(k.window for k in rp.cache.paged_keys) == [9, 20]
    check_close(np.concatenate(rows), ref, "float32", "a request longer than its pools", k=KP["float32"])
    rp.step([], ["x"])
    assert rp.cache.live == 0 and all(rp.cache.free_pages(g) == rp.cache.group_pages[g] for g in range(len(rp.cache.group_pages)))


# ------------------------------------------------------------------------------------- window edges, far keys, sinks
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sharp_attention_at_the_edges_and_far_back(tmp_path, dtype):
    """A softmax so peaked that a row's output is a few single keys wherever they lie: a key lost at a page border or at the
    edge of the window, or one seen from just outside it, changes the logits outright. The test first asserts, on the plain
    model, that such rows exist."""
    window = 45
    sharp = 5.0 if dtype == "float32" else 2.0
    config = model_config(128, 64, [lat2(4, 16, 16, 32, 32, window=window, scale=0.15 * sharp), lat(4, 16, 16, 16, 32, rot=(10000.0, 16, yarn(2.0, 256)), scale=0.12 * sharp),
                                    lat2(2, 32, 16, 48, 24, window=100, scale=0.1 * sharp)])
    from cellm_b200.weights import InitSpec
    folder = write_model(tmp_path / "sharp", config, 9, init=InitSpec(linear_std=0.25, embedding_std=0.8, bias_std=0.05, norm_jitter=0.1))
    cfg, w = load_plain(folder)
    rng = np.random.default_rng(4)
    toks = rng.integers(0, cfg["vocab"], 500).tolist()
    reqs = {"long": toks, "short": toks[:46]}
    ref = {rid: Ref(t, cfg, w, runs=4) for rid, t in reqs.items()}
    eps, pos = cfg["norm"]["eps"], torch.arange(len(toks))
    x0 = w["embed"][torch.tensor(toks)]
    h0 = plain.rms_norm(x0, w["l0.norm1"], eps)
    seen, wide = [], []
    y = plain.latent_attention_2(h0, w, "l0.mix.", cfg["layers"][0]["mixer"], eps, seen)
    plain.latent_attention_2(h0, w, "l0.mix.", {**cfg["layers"][0]["mixer"], "mask": {"size": window + 1}}, eps, wide)
    top, where = seen[0][:, 100:].max(-1)
    assert float(top.median()) > (0.5 if dtype == "float32" else 0.25)
    rows = torch.arange(100, 500)[None]
    assert int((rows - where == window - 1).sum()) >= 3          # the heaviest key is the last one the window keeps
    assert int((wide[0][:, 100:].gather(2, (rows - window).expand(4, -1)[..., None]) > 0.5).sum()) >= 2      # the next one would win
    x1 = x0 + plain.rms_norm(y, w["l0.norm1b"], eps)
    seen = []
    plain.latent_attention(plain.rms_norm(x1, w["l1.norm1"], eps), w, "l1.mix.", cfg["layers"][1]["mixer"], pos, eps, seen)
    top, where = seen[0][:, 400:].max(-1)
    assert float(top.median()) > 0.2 and float((torch.arange(400, 500)[None] - where).float().median()) > 60      # reaches far back
    for fam in ("whole", "tail", "portions", "mixed"):
        for page in (8, 32):
            got = run_trace(folder, dtype, FAMILIES[fam](reqs), page)
            for rid, t in reqs.items():
                # so peaked a softmax passes a score's last bits on; a lost or surplus key moves a row by a tenth of the
                # logits' size and more
                against_plain(traces.as_matrix(got[rid], len(t)), ref[rid], dtype, f"sharp {dtype} {fam} page {page} {rid}", k32=1e-4)


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sinks_and_gates_decide(tmp_path, dtype):
    """Sinks far above, among and far below the scores, and gates from nearly shut to open: the plain logits move outright when
    either is left out, and the engine's follow."""
    config = model_config(90, 64, [lat2(4, 16, 16, 32, 32, window=30), lat(4, 16, 16, 16, 48, rot=(500.0, 16))])
    folder = write_model(tmp_path / "s", config, 12)
    from cellm_b200.weights.safetensors_io import SafetensorsFile, save_file
    path = os.path.join(folder, "model.safetensors")
    sf = SafetensorsFile(path)
    tensors = {n: sf.tensor(n).clone() for n in sf.names()}
    sf.close()
    tensors["l0.mix.sink"] = torch.tensor([9.0, 1.5, 0.0, -60.0]).to(tensors["l0.mix.sink"].dtype)
    tensors["l1.mix.g"] *= 4
    save_file(tensors, path, {"format": "pt"})
    cfg, w = load_plain(folder)
    toks = np.random.default_rng(3).integers(0, 90, 150).tolist()
    reqs = {"x": toks, "y": toks[40:43]}
    ref = {rid: Ref(t, cfg, w) for rid, t in reqs.items()}
    for without in ({"l0.mix.sink": torch.full((4,), -1e4, dtype=torch.float64)}, {"l1.mix.g": torch.zeros(4, 64, dtype=torch.float64)}):
        other = plain.forward(toks, cfg, {**w, **without}).numpy()
        assert np.median(np.abs(other - ref["x"]).max(axis=1)) > 0.1 * np.abs(ref["x"]).max()
    for fam in FAMILIES:
        got = run_trace(folder, dtype, FAMILIES[fam](reqs), 8)
        for rid, t in reqs.items():
            against_plain(traces.as_matrix(got[rid], len(t)), ref[rid], dtype, f"sinks and gates {dtype} {fam} {rid}")


# ------------------------------------------------------------------------------------------ generation
def check_greedy_tokens(cfg, w, prompt, out, dtype):
    seq = list(prompt) + list(out[:-1])
    ref = plain.forward(seq, cfg, w)[len(prompt) - 1:].numpy()
    tol = 2 * KP[dtype] * (1 + np.abs(ref).max())
    for j, t in enumerate(out):
        best = int(ref[j].argmax())
        assert t == best or ref[j][best] - ref[j][t] <= tol, f"token {j}: {t} where the plain model has {best}"


@pytest.mark.parametrize("name,dtype", [("a", "float32"), ("d", "float32"), ("c", "bfloat16")])
def test_greedy_generation_through_the_engine(models, name, dtype):
    from cellm_b200 import Engine, SamplingParams
    folder, reqs, _ = models[name]
    cfg, w = load_plain(folder)
    prompts = [t for t in reqs.values() if len(t) < 140][:5]
    eng = Engine(folder, dtype=dtype, tokens_per_block=8, total_blocks=96, max_num_seqs=3, max_batch_tokens=48, prefill_chunk=24)
    outs = eng.generate(prompts, SamplingParams.greedy(14, stop_eos=False))
    for prompt, out in zip(prompts, outs):
        assert len(out) == 14
        check_greedy_tokens(cfg, w, prompt, out, dtype)
    again = eng.generate(prompts[:2], SamplingParams.greedy(14, stop_eos=False))      # slots and pages used again
    for prompt, out in zip(prompts[:2], again):
        check_greedy_tokens(cfg, w, prompt, out, dtype)
    s = eng.stats()
    assert s["idle"] and s["free_pages"] == s["total_pages"] and s["free_slots"] == 3


def test_the_command_lines_run_the_design(models, tmp_path):
    folder, reqs, ref = models["b"]
    env = {**os.environ, "PYTHONPATH": ROOT}
    prompt = reqs["r3"]
    p = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "infer"), "--model", folder, "--tokens", ",".join(map(str, prompt)),
                        "--gen", "6", "--temperature", "0", "--dtype", "float32", "--stop-eos", "false"], capture_output=True, text=True,
                       env=env, timeout=600)
    assert p.returncode == 0, p.stderr[-2000:]
    cfg, w = load_plain(folder)
    out = [int(t) for t in re.search(r"^tokens: ([\d,]+)$", p.stdout, re.M).group(1).split(",")]
    assert len(out) == 6
    check_greedy_tokens(cfg, w, prompt, out, "float32")
    steps = traces.portions({"r3": prompt}, (7, 2, 4))
    q = subprocess.run([sys.executable, os.path.join(ROOT, "bin", "trace_run"), "--model", folder, "--dtype", "float32", "--out",
                        str(tmp_path / "o"), "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n",
                       capture_output=True, text=True, env=env, timeout=600)
    assert q.returncode == 0, q.stderr[-2000:]
    assert [l for l in q.stdout.splitlines() if l.startswith("done")] == [f"done {i}" for i in range(len(steps))]
    rows = np.concatenate([np.fromfile(tmp_path / "o" / f"{i}.f32", dtype="<f4").reshape(-1, cfg["vocab"]) for i in range(len(steps))])
    check_close(rows, ref["r3"], "float32", "trace_run", k=KP["float32"])


# ------------------------------------------------------------------------------------- the mechanisms by themselves
def step_ctx(q_lens, ctx_lens, slots=None, dtype=torch.float32):
    """A step's index arrays for requests that bring q_lens[b] tokens after ctx_lens[b] earlier ones."""
    from cellm_b200.ops._state import error_word
    from cellm_b200.parts.base import StepContext
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    T, B = sum(q_lens), len(q_lens)
    pos = [c + i for c, n in zip(ctx_lens, q_lens) for i in range(n)]
    seq = [b for b, n in enumerate(q_lens) for _ in range(n)]
    return StepContext(T=T, B=B, dtype=dtype, device=torch.device(DEV), token_ids=i32([0] * T), positions=i32(pos), seq_of_token=i32(seq),
                       cu_seqlens=i32([0] + list(np.cumsum(q_lens))), ctx_lens=i32(ctx_lens), slot_ids=i32(slots or list(range(B))),
                       err=error_word(torch.device(DEV)), q_lens=list(q_lens), ctx_lens_host=list(ctx_lens), max_q_len=max(q_lens),
                       max_total_len=max(c + n for c, n in zip(ctx_lens, q_lens)))


def paged(lens, kw, page, dtype, g, fill=0.0):
    """(binding, pages of each request): one pool whose pages the requests hold in an order of their own."""
    from cellm_b200.parts.base import CacheBinding
    width = max(-(-n // page) for n in lens) + 1
    n_pages = len(lens) * width + 3
    order = torch.randperm(n_pages, generator=g).tolist()
    table = torch.full((len(lens), width), -1, dtype=torch.int32)
    for b, n in enumerate(lens):
        for i in range(-(-n // page)):
            table[b, i] = order.pop()
    pool = torch.full((n_pages, 1, page, kw), fill, dtype=dtype, device=DEV)
    return CacheBinding(k=pool, block_table=table.to(DEV), page_size=page, num_pages=n_pages), table


MIXERS = {  # params beside the sizes H, heads, dim, rot_dim, vdim, rank
    "gated": ((40, 4, 16, 8, 12, 24), {"gate": True, "rot": (100.0, 8)}),
    "gated, stretched": ((64, 2, 32, 32, 32, 64), {"gate": True, "rot": (10000.0, 32, yarn(8.0, 64, 8.0, 2.0))}),
    "gated, part of it turned": ((48, 3, 10, 6, 5, 16), {"gate": True, "rot": (50.0, 4)}),
    "gated, no rotated part": ((33, 5, 7, 0, 9, 16), {"gate": True}),
    "latent queries, window, sinks": ((40, 4, 16, 0, 12, 32), {"q_rank": 20, "window": 17, "sinks": True}),
    "latent queries of odd sizes": ((33, 3, 5, 0, 7, 11), {"q_rank": 9, "window": 1, "sinks": True}),
    "latent queries, every row": ((64, 2, 32, 0, 64, 128), {"q_rank": 48, "sinks": True}),
    "all of it": ((72, 3, 8, 8, 16, 48), {"q_rank": 24, "window": 30, "sinks": True, "gate": True, "rot": (300.0, 8, yarn(2.0, 128))}),
    "all of it, odd": ((50, 2, 9, 6, 16, 26), {"q_rank": 7, "window": 23, "sinks": True, "gate": True, "rot": (300.0, 6)}),
    "gated, interleaved pairs": ((40, 2, 8, 8, 8, 24), {"gate": True, "rot": (100.0, 8), "layout": "interleaved"}),
}


def plain_mixer(h, w, sizes, opt, eps):
    """Every form of the mixer from the plain pieces."""
    H, nh, d, r, vd, rank = sizes
    T, pos = h.shape[0], torch.arange(h.shape[0])
    q = plain.lin(plain.rms_norm(plain.lin(h, w["dq"]), w["dq_norm"], eps), w["uq"]) if opt.get("q_rank") else plain.lin(h, w["q"])
    q, down = q.view(T, nh, d + r), plain.lin(h, w["dkv"])
    c = plain.rms_norm(down[:, :rank], w["dkv_norm"], eps)
    k, v = plain.lin(c, w["uk"]).view(T, nh, d), plain.lin(c, w["uv"]).view(T, nh, vd)
    s = torch.einsum("ihd,jhd->hij", q[..., :d], k)
    if r:
        rot = opt.get("rot")
        rot = None if rot is None else {"base": rot[0], "dims": rot[1], **({"scaling": rot[2]} if len(rot) > 2 else {})}

        def turn(x):
            if opt.get("layout") != "interleaved":
                return plain.turn(x, pos, rot)
            n = rot["dims"]
            apart = torch.cat([x[..., 0:n:2], x[..., 1:n:2], x[..., n:]], dim=-1)
            t = plain.turn(apart, pos, rot)
            back = t.clone()
            back[..., 0:n:2], back[..., 1:n:2] = t[..., :n // 2], t[..., n // 2:n]
            return back
        s = s + torch.einsum("ihd,jd->hij", turn(q[..., d:]), turn(down[:, rank:]))
    pr = plain.weights_of_scores(s * opt["scale"], plain.visible(T, opt.get("window")), w["sinks"] if opt.get("sinks") else None)
    o = torch.einsum("hij,jhd->ihd", pr, v)
    if opt.get("gate"):
        o = o * torch.sigmoid(plain.lin(h, w["g"]))[:, :, None]
    return plain.lin(o.reshape(T, nh * vd), w["o"])


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("name", list(MIXERS))
def test_mixer_alone(name, dtype):
    """Two sequences side by side in pages of their own, whole, in portions down to one token and token by token."""
    from cellm_b200.config.plan import PartSpec
    from cellm_b200.parts.latent_attention import LatentAttentionMixer
    sizes, opt = MIXERS[name]
    H, nh, d, r, vd, rank = sizes
    g = torch.Generator().manual_seed(H * 10 + nh)
    rnd = lambda *s: torch.randn(*s, generator=g)
    qr, eps = opt.get("q_rank", 0), 1e-5
    w = {"dkv": rnd(rank + r, H) / H ** 0.5, "dkv_norm": 1 + 0.2 * rnd(rank), "uk": rnd(nh * d, rank) / rank ** 0.5, "uv": rnd(nh * vd, rank) / rank ** 0.5,
         "o": rnd(H, nh * vd) / (nh * vd) ** 0.5}
    if qr:
        w.update(dq=rnd(qr, H) / H ** 0.5, dq_norm=1 + 0.2 * rnd(qr), uq=rnd(nh * (d + r), qr) / qr ** 0.5)
    else:
        w["q"] = rnd(nh * (d + r), H) / H ** 0.5
    if opt.get("sinks"):
        w["sinks"] = torch.linspace(-2.0, 3.0, nh)
    if opt.get("gate"):
        w["g"] = 2 * rnd(nh, H) / H ** 0.5
    opt = {**opt, "scale": 1.3 * (d + r) ** -0.5}
    w = {k: v.to(dtype) for k, v in w.items()}
    rope = None if "rot" not in opt else PartSpec("rope", {"head_dim": r, "rotary_dim": opt["rot"][1], "theta": opt["rot"][0], "layout": opt.get("layout", "half"),
                                                           "scaling": opt["rot"][2] if len(opt["rot"]) > 2 else None})
    params = {"hidden_size": H, "heads": nh, "dim": d, "rot_dim": r, "vdim": vd, "kv_rank": rank, "scale": opt["scale"], "eps": eps, "position": rope,
              "window": opt.get("window", 0), "sinks": bool(opt.get("sinks")), "q_rank": qr, "gate": bool(opt.get("gate"))}
    part = LatentAttentionMixer(params, {k: v.to(DEV) for k, v in w.items()}, dtype)
    lens = [90, 31]
    x = [rnd(n, H).to(dtype) for n in lens]
    want = [plain_mixer(t.double(), {k: v.double() for k, v in w.items()}, sizes, opt, eps) for t in x]
    for cut in ((128,), (5, 1, 2, 11, 30), (1,)):
        cache, _ = paged(lens, rank + r, 8, dtype, g)
        got, fed, k = [[], []], [0, 0], 0
        while any(f < n for f, n in zip(fed, lens)):
            live = [b for b in range(2) if fed[b] < lens[b]]
            n = [min(cut[k % len(cut)], lens[b] - fed[b]) for b in live]
            k += 1
            ctx = step_ctx(n, [fed[b] for b in live], dtype=dtype)
            o = part.forward(torch.cat([x[b][fed[b]:fed[b] + m] for b, m in zip(live, n)]).to(DEV), ctx,
                             replace(cache, block_table=cache.block_table[live].contiguous())).cpu().double()
            at = 0
            for b, m in zip(live, n):
                got[b].append(o[at:at + m])
                at, fed[b] = at + m, fed[b] + m
        for b in range(2):
            size = float(want[b].abs().max())
            tol = dict(rtol=1e-4, atol=2e-5 * size) if dtype == torch.float32 else dict(rtol=3e-2, atol=3e-2 * size)
            torch.testing.assert_close(torch.cat(got[b]), want[b], msg=lambda m: f"{name} {cut} sequence {b}: {m}", **tol)
    assert int(ctx.err.item()) == 0


@pytest.mark.parametrize("nh,kw,dv,page,window", [(8, 80, 64, 16, 0), (4, 96, 96, 32, 50), (5, 48, 32, 8, 33), (3, 64, 48, 16, 1), (2, 576, 512, 16, 70), (3, 144, 128, 64, 64)])
def test_latent_kernel_with_gates_and_sinks(nh, kw, dv, page, window):
    """The tensor-core kernel alone, whole and with the keys in pieces (gate and sink are then the merge's): prompt portions and
    decoded tokens at contexts that end inside a page and inside a block of keys, against 64-bit torch over the same rounded
    inputs."""
    from cellm_b200 import ops
    g = torch.Generator().manual_seed(nh * 1000 + kw)
    q_lens, ctx_lens = [70, 1, 9, 1], [131, 300, 0, 63]
    T = sum(q_lens)
    cache, table = paged([c + n for c, n in zip(ctx_lens, q_lens)], kw, page, torch.bfloat16, g)
    pool = (torch.randn(cache.k.shape, generator=g) * 0.7).to(torch.bfloat16)
    q = (torch.randn(T, nh * kw, generator=g) * 0.7).to(torch.bfloat16)
    gate, sinks = torch.randn(T, nh, generator=g) * 3, torch.linspace(-3.0, 4.0, nh)
    scale = 1.7 * kw ** -0.5
    want = torch.zeros(T, nh, dv, dtype=torch.float64)
    t = 0
    for b, n in enumerate(q_lens):
        rows = torch.stack([pool[table[b, j // page], 0, j % page] for j in range(ctx_lens[b] + n)]).double()
        for i in range(n):
            hi = ctx_lens[b] + i + 1
            lo = max(0, hi - window) if window else 0
            s = (q[t].double().reshape(nh, kw) @ rows[lo:hi].T) * scale
            top = torch.maximum(s.amax(-1), sinks.double())[:, None]
            e = torch.exp(s - top)
            want[t] = (e / (e.sum(-1, keepdim=True) + torch.exp(sinks.double()[:, None] - top))) @ rows[lo:hi, :dv]
            t += 1
    want = want * torch.sigmoid(gate.double())[:, :, None]
    ctx = step_ctx(q_lens, ctx_lens)
    for nsplit in (1, 3, 8):
        out = ops.attention_latent(q.to(DEV), pool.to(DEV), ctx.cu_seqlens, ctx.ctx_lens, cache.block_table, q_lens, nh, dv, scale, nsplit, ctx.err,
                                   window, sinks.to(DEV), gate.to(DEV))
        torch.testing.assert_close(out.cpu().double().reshape(T, nh, dv), want, rtol=2e-2, atol=1e-2)
    assert int(ctx.err.item()) == 0


EXPANDED = [  # heads, dim, rot_dim, vdim, rank
    (4, 128, 64, 128, 512), (2, 64, 0, 64, 64), (3, 16, 16, 16, 24), (2, 48, 32, 80, 40), (1, 96, 64, 112, 128), (2, 192, 64, 128, 64), (5, 32, 0, 32, 96),
    (2, 128, 0, 48, 72), (1, 64, 96, 96, 16),
]


@pytest.mark.parametrize("window", [0, 1, 50, 128, 129, 300])
@pytest.mark.parametrize("heads,dim,rot,vdim,rank", EXPANDED)
def test_expanded_attention_alone(heads, dim, rot, vdim, rank, window):
    """The tcgen05 attention over keys and values that were expanded from the rows: portions of several requests (one with a single
    token, one with none) at contexts that end inside a block of keys, at its edge and inside a page; tiles that start inside a
    block and blocks that only one of a pair of tiles reads; sinks and gates. Against 64-bit torch over the same rounded
    inputs. The rows themselves come out of pages in an order of their own, those behind the window taken away."""
    from cellm_b200 import ops
    g = torch.Generator().manual_seed(heads * 1000 + dim + vdim)
    q_lens, ctx_lens, page = [300, 1, 129, 0, 256, 7, 520], [0, 40, 131, 20, 128, 500, 255], 16
    T, kw = sum(q_lens), rank + rot
    rnd = lambda *s: (torch.randn(*s, generator=g) * 0.7).to(torch.bfloat16)
    cache, table = paged([c + n for c, n in zip(ctx_lens, q_lens)], kw, page, torch.bfloat16, g)
    pool = rnd(*cache.k.shape)
    first = [max(0, c - window + 1) if window else 0 for c in ctx_lens]
    bt = cache.block_table.clone()
    for b, f in enumerate(first):
        bt[b, :f // page] = -1
    ctx = step_ctx(q_lens, ctx_lens)
    keep = [range(f, c + n) if n else [] for f, c, n in zip(first, ctx_lens, q_lens)]
    n_rows = sum(len(k) for k in keep)
    rows = ops.latent_rows(pool.to(DEV), ctx.cu_seqlens, ctx.ctx_lens, bt, n_rows, ctx.err, window)
    want_rows = torch.cat([torch.stack([pool[table[b, j // page], 0, j % page] for j in k]) for b, k in enumerate(keep) if len(k)])
    assert torch.equal(rows.cpu(), want_rows)
    qw = dim + rot
    q, q_rot, kv = rnd(T, heads * qw + 8), rnd(T, heads * rot) if rot else None, rnd(n_rows, heads * (dim + vdim))
    sinks, gate = torch.linspace(-2.0, 3.0, heads), torch.randn(T, heads, generator=g) * 2
    scale = 1.5 * qw ** -0.5
    for with_extras in (True, False):
        want, t, at = torch.zeros(T, heads, vdim, dtype=torch.float64), 0, 0
        for b, n in enumerate(q_lens):
            m = len(keep[b])
            if not n:
                continue
            k = kv[at:at + m, :heads * dim].double().view(m, heads, dim)
            v = kv[at:at + m, heads * dim:].double().view(m, heads, vdim)
            qq = q[t:t + n, :heads * qw].double().view(n, heads, qw)[..., :dim]
            s = torch.einsum("ihd,jhd->hij", qq, k)
            if rot:
                s = s + torch.einsum("ihd,jd->hij", q_rot[t:t + n].double().view(n, heads, rot), rows[at:at + m, rank:].cpu().double())
            back = (ctx_lens[b] + torch.arange(n))[:, None] - (first[b] + torch.arange(m))[None, :]
            sees = (back >= 0) & ((back < window) if window else (back >= 0))
            pr = plain.weights_of_scores(s * scale, sees, sinks.double() if with_extras else None)
            want[t:t + n] = torch.einsum("hij,jhd->ihd", pr, v)
            t, at = t + n, at + m
        if with_extras:
            want = want * torch.sigmoid(gate.double())[:, :, None]
        out = ops.attention_expanded(q.to(DEV), q_rot.to(DEV) if rot else None, rows, kv.to(DEV), ctx.cu_seqlens, ctx.ctx_lens, q_lens, heads, dim, rot, vdim,
                                     scale, ctx.err, window, sinks.to(DEV) if with_extras else None, gate.to(DEV) if with_extras else None)
        assert int(ctx.err.item()) == 0
        torch.testing.assert_close(out.cpu().double().view(T, heads, vdim), want, rtol=2e-2, atol=1e-2)


def test_expanded_attention_refuses_what_it_does_not_take():
    from cellm_b200.ops import _lib
    supports = _lib.fn("attention_expanded", "cellm_attention_expanded_supports")
    assert all(supports(*s) for s in EXPANDED)
    assert not any(supports(*s) for s in [(2, 24, 0, 16, 16), (2, 16, 8, 16, 16), (2, 16, 0, 20, 16), (2, 16, 0, 144, 16), (2, 16, 0, 16, 12), (2, 320, 0, 64, 64), (0, 16, 0, 16, 16)])


@pytest.mark.parametrize("windows", [(0, 90), (40, 0)])
def test_expanded_portions_against_the_rows_themselves(tmp_path, windows):
    """Whole models whose prompt portions take the expanded form, against the plain model and against the same engine with the form
    switched off: prompts of several tiles, portions that start inside a block, portions beside single tokens, requests that
    share a step."""
    from cellm_b200.runtime import program
    config = model_config(200, 128, [lat2(4, 32, 48, 64, 64, window=windows[0], mlp=moe(4, 2, 64, 1.0, (2, 1), (64, 1.5))),
                                     lat(2, 64, 32, 64, 128, rot=(1000.0, 32, yarn(2.0, 128))), lat2(2, 48, 32, 96, 40, window=windows[1])])
    folder = write_model(tmp_path / "m", config, 6)
    cfg, w = load_plain(folder)
    rng = np.random.default_rng(5)
    reqs = {"x": rng.integers(0, 200, 700).tolist(), "y": rng.integers(0, 200, 333).tolist(), "z": rng.integers(0, 200, 40).tolist()}
    ref = {rid: Ref(t, cfg, w) for rid, t in reqs.items()}
    assert min(r.margin for r in ref.values()) > 0.1
    both = [{"step": 0, "entries": [{"id": r, "tokens": t[:n], "want": list(range(n))} for (r, t), n in zip(reqs.items(), (300, 200, 39))], "end": []},
            {"step": 1, "entries": [{"id": r, "tokens": t[a:b], "want": list(range(b - a))} for (r, t), a, b in zip(reqs.items(), (300, 200, 39), (699, 333, 40))],
             "end": ["y", "z"]},
            {"step": 2, "entries": [{"id": "x", "tokens": reqs["x"][699:], "want": [0]}], "end": ["x"]}]
    old = dict(program.OPTIONS)
    outs = {}
    try:
        program.OPTIONS["attention_tc_min_ctas"] = 1
        for on in (True, False):
            program.OPTIONS["latent_expand"] = on
            before = program.CALLS["cellm_attention_expanded"]
            outs[on] = {"whole": run_trace(folder, "bfloat16", traces.whole(reqs), 16),
                        "portions": run_trace(folder, "bfloat16", traces.portions(reqs, (300, 130, 2, 190)), 8), "both": run_trace(folder, "bfloat16", both, 16)}
            assert (program.CALLS["cellm_attention_expanded"] > before) == on
    finally:
        program.OPTIONS.update(old)
    for fam in outs[True]:
        for rid, t in reqs.items():
            got = traces.as_matrix(outs[True][fam][rid], len(t))
            against_plain(got, ref[rid], "bfloat16", f"expanded {fam} {rid}")
            check_close(got, traces.as_matrix(outs[False][fam][rid], len(t)), "bfloat16", f"expanded vs rows, {fam} {rid}", k=K_SELF["bfloat16"])


@pytest.mark.parametrize("window,page", [(0, 8), (1, 4), (16, 8), (21, 8), (33, 16), (130, 32), (400, 16)])
@pytest.mark.parametrize("kw,dv", [(24, 8), (32, 16), (80, 64)])
def test_a_window_sees_exactly_its_rows(window, page, kw, dv):
    """One row's values name its place; a query scores every row alike, so the output tells which rows were summed: the window's
    last ones up to the token itself. Prompt rows and single decoded rows with the pages behind the window taken away, in
    32-bit and on the tensor cores, through the mixer's attention alone."""
    from cellm_b200 import ops
    g = torch.Generator().manual_seed(window * 100 + page)
    T, nh = 150, 2
    place = torch.arange(T)
    for dtype in (torch.float32, torch.bfloat16):
        if dtype == torch.bfloat16 and kw % 16:
            continue
        cache, table = paged([T], kw, page, dtype, g, fill=5.0)
        rows = torch.zeros(T, kw)
        rows[:, 0], rows[:, 1], rows[:, 2], rows[:, kw - 1] = place % 8, (place // 8) % 8, place // 64, 1.0
        for j in range(T):
            cache.k[table[0, j // page], 0, j % page] = rows[j].to(dtype).to(DEV)
        q = torch.zeros(T, nh, kw)
        q[:, :, kw - 1] = 0.5
        edges = [0, T - 1, page - 1, page, window - 1, window, window + 1, 2 * window]
        for some in [list(range(T))] + [[r] for r in edges]:
            some = [r for r in some if 0 <= r < T]
            if not some:
                continue
            single = len(some) == 1
            ctx = step_ctx([1], [some[0]]) if single else step_ctx([T], [0])
            bt = cache.block_table.clone()
            if single and window:
                bt[0, :max(0, some[0] - window + 1) // page] = -1
            qq = q[some].reshape(len(some), -1).to(dtype).to(DEV).contiguous()
            if dtype == torch.float32:
                out = ops.attention_plain_masked(qq, replace(cache, block_table=bt), ctx, nh, 1, kw, dv, 1.0, window)
            else:
                out = ops.attention_latent(qq, cache.k, ctx.cu_seqlens, ctx.ctx_lens, bt, ctx.q_lens, nh, dv, 1.0, 1 if not single else 3, ctx.err, window)
            out = out.cpu().double().reshape(len(some), nh, dv)
            assert int(ctx.err.item()) == 0
            tol = 1e-4 if dtype == torch.float32 else 6e-3
            for n, i in enumerate(some):
                seen = place[(place <= i) & ((place > i - window) if window else (place >= 0))]
                for c, digit in enumerate((seen % 8, (seen // 8) % 8, seen // 64)):
                    mean = float(digit.double().mean())
                    assert abs(float(out[n, 1, c]) - mean) <= tol * (1 + mean), (dtype, i, c)


@pytest.mark.parametrize("T,H", [(9, 54), (5, 56), (3, 2048), (70, 1100), (2, 4096), (2, 8192), (2, 9000), (4, 512), (1, 8)])
def test_norm_sum_and_norm_alone(T, H):
    """The addend's norm, the sum into the stream and the next norm as one kernel: all rows, and some rows without touching the
    stream; addends of very different sizes, an eps that matters."""
    from cellm_b200 import ops
    g = torch.Generator().manual_seed(T * 7 + H)
    rnd = lambda *s: torch.randn(*s, generator=g)
    x, a, w1, w2 = rnd(T, H) * 3 + 0.5, rnd(T, H) * torch.logspace(-3, 2, T)[:, None], 1 + 0.2 * rnd(H), 1 + 0.2 * rnd(H)
    rows = torch.tensor([T - 1, 0, T // 2], dtype=torch.int32)
    for act, wd in ((torch.float32, torch.float32), (torch.float32, torch.bfloat16), (torch.bfloat16, torch.bfloat16), (torch.bfloat16, torch.float32)):
        ad, v1, v2 = a.to(act), w1.to(wd), w2.to(wd)
        sum_ = x.double() + plain.rms_norm(ad.double(), v1.double(), 1e-3)
        want = plain.rms_norm(sum_, v2.double(), 1e-5)
        tol = dict(rtol=1e-5, atol=1e-5) if act == torch.float32 else dict(rtol=8e-3, atol=8e-3)
        xd = x.to(DEV).clone()
        y = ops.norm_add_norm(xd, ad.to(DEV), v1.to(DEV), 1e-3, v2.to(DEV), 1e-5, rows.to(DEV))
        assert torch.equal(xd.cpu(), x)
        torch.testing.assert_close(y.cpu().double(), want[rows.long()], **tol)
        y = ops.norm_add_norm(xd, ad.to(DEV), v1.to(DEV), 1e-3, v2.to(DEV), 1e-5)
        assert y.dtype == act
        torch.testing.assert_close(xd.cpu().double(), sum_, rtol=1e-5, atol=1e-5)
        torch.testing.assert_close(y.cpu().double(), want, **tol)


def test_norms_behind_follow_their_products_at_once(tmp_path):
    """A step launched without a pause between its kernels gives what the same step gives with the host waiting after each part:
    the fused norm's loads stay behind the kernels that produce what it reads."""
    from cellm_b200.models import load_model
    from cellm_b200.parts import block as B
    from cellm_b200.replay import Replayer
    config = model_config(300, 512, [lat2(4, 32, 32, 64, 64, window=20, mlp=moe(8, 2, 64, 1.0, (4, 2), (64, 1.0))) for _ in range(6)])
    folder = write_model(tmp_path / "m", config, 2)
    toks = np.random.default_rng(0).integers(0, 300, 60).tolist()
    loaded = load_model(folder, "bfloat16")
    outs = []
    for by_parts in (False, True, False):
        emit = B.SandwichNormBlock.emit
        if by_parts:
            B.SandwichNormBlock.emit = B.Block.emit
        try:
            loaded[2].program = None
            rp = Replayer(loaded, "bfloat16", 64, 8, 4, use_graphs=False)
            rows = [rp.step([{"id": "x", "tokens": toks[:40], "want": list(range(40))}], [])]
            rows += [rp.step([{"id": "x", "tokens": [t], "want": [0]}], []) for t in toks[40:]]
            outs.append(np.concatenate(rows))
        finally:
            B.SandwichNormBlock.emit = emit
            loaded[2].program = None
    assert np.array_equal(outs[0], outs[2])
    check_close(outs[0], outs[1], "bfloat16", "at once vs part by part", k=K_SELF["bfloat16"])


def test_soft_cap_alone():
    from cellm_b200 import ops
    g = torch.Generator().manual_seed(0)
    for n, cap in ((1, 3.0), (7, 30.0), (1024, 5.0), (3 * 4001, 50.0)):
        z = torch.randn(n, generator=g) * torch.logspace(-2, 3, n)
        got = ops.soft_cap_(z.to(DEV).clone(), cap).cpu().double()
        torch.testing.assert_close(got, cap * torch.tanh(z.double() / cap), rtol=2e-6, atol=1e-7)
        assert float(got.abs().max()) <= cap


def test_softmax_over_all_within_groups():
    """The router alone against the plain choice: runs of neighbours scored by their largest, weights over their own sum, ties to
    the lower index, sums far from zero, one expert a group, one group, more kept than needed."""
    from cellm_b200.ops._lib import fn, ptr, stream_of
    g = torch.Generator().manual_seed(2)
    for E, top, n, keep in ((8, 3, 4, 2), (6, 1, 3, 1), (12, 5, 2, 2), (1, 1, 1, 1), (64, 6, 8, 4), (5, 5, 1, 1), (16, 4, 16, 5), (100, 7, 4, 3), (256, 8, 8, 4)):
        T = 41
        z = torch.randn(T, E + 1, generator=g) * 2
        z[3, :E] = 0.0
        z[4, :E] += 300.0
        z[5, :E] -= 300.0
        z[6, 0] = 60.0                                                     # one score takes nearly all of the sum
        for bias in (None, torch.randn(E, generator=g)):
            idx = torch.empty(T, top, dtype=torch.int32, device=DEV)
            wts, gate = torch.empty(T, top, device=DEV), torch.empty(T, device=DEV)
            zd, bd = z.to(DEV), None if bias is None else bias.to(DEV)
            assert fn("kernels_common", "cellm_route_softmax_all")(ptr(idx), ptr(wts), ptr(gate), ptr(zd), E + 1, ptr(bd), 0, T, E, top, n, keep, 1.0, 1,
                                                                   stream_of(zd)) == 0
            s = z[:, :E] + (bias if bias is not None else 0.0)
            want_idx, want_w = plain.route(s.double(), top, {"count": n, "keep": keep})
            assert torch.equal(idx.cpu().long(), want_idx), (E, top, n, keep)
            torch.testing.assert_close(wts.cpu().double(), want_w, rtol=2e-5, atol=1e-6)
            torch.testing.assert_close(gate.cpu().double(), torch.sigmoid(z[:, E].double()), rtol=1e-5, atol=1e-7)
    assert fn("kernels_common", "cellm_route_softmax_all")(ptr(idx), ptr(wts), ptr(gate), ptr(zd), 9, None, 0, 4, 8, 5, 4, 2, 1.0, 0, stream_of(zd)) == -2


MIXTURES = [  # H, experts, top, ff, limit, groups, (shared ff, limit)
    (96, 12, 4, 40, 0.7, (4, 2), (56, 1.2)), (54, 5, 4, 21, 1.5, None, (33, 0.4)), (128, 16, 1, 64, 0.9, (8, 3), None), (64, 8, 8, 32, 2.0, (2, 2), (16, 2.0)),
    (2048, 64, 6, 256, 1.0, (8, 4), (512, 0.8)), (104, 6, 2, 24, None, (3, 1), (8, None)), (256, 32, 3, 128, 1.1, (4, 4), None), (64, 1, 1, 70, 0.5, None, (20, 3.0)),
    (72, 3, 2, 192, 0.3, (3, 2), (128, 0.6)),
]


@pytest.mark.parametrize("T", [1, 5, 16, 17, 150, 300])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,E,top,ff,limit,groups,shared", MIXTURES)
def test_clamped_experts_against_plain(dtype, T, H, E, top, ff, limit, groups, shared):
    """The part alone on random inputs whose gates and ups lie on both sides of both limits. Few tokens take the row-by-row
    kernels, many (under bfloat16, with widths the tensor cores take) the grouped products. Rows whose choice is close in
    32-bit are given up to that."""
    from cellm_b200.parts.routed_experts import RoutedExperts
    if H == 2048 and T not in (5, 150):
        pytest.skip("the large shape at two sizes")
    g = torch.Generator().manual_seed(H * 7 + E)
    rnd = lambda *s: torch.randn(*s, generator=g)
    w = {"router": rnd(E, H) * 3 / H ** 0.5}
    for e in range(E):
        w[f"gate_{e}"], w[f"up_{e}"], w[f"down_{e}"] = rnd(ff, H) / H ** 0.5, rnd(ff, H) / H ** 0.5, rnd(H, ff) / ff ** 0.5
    params = {"hidden_size": H, "experts": E, "top": top, "ff_dim": ff, "activation": "clamped", "limit": limit, "slope": 1.702, "scores": "softmax_all",
              "gated": True, "correction": False, "groups": groups[0] if groups else 1, "keep_groups": groups[1] if groups else 1}
    m = {"router": {"experts": E, "top": top, **({"groups": {"count": groups[0], "keep": groups[1]}} if groups else {})}, "expert": {"ff": ff, "limit": limit}}
    if shared:
        w.update(shared_gate_proj=rnd(shared[0], H) / H ** 0.5, shared_up=rnd(shared[0], H) / H ** 0.5, shared_down=rnd(H, shared[0]) / shared[0] ** 0.5)
        params.update(shared_ff=shared[0], shared_limit=shared[1], shared_gate=False)
        m["shared"] = {"ff": shared[0], "limit": shared[1]}
    w = {k: v.to(dtype).to(DEV) for k, v in w.items()}
    x = rnd(T, H).to(dtype).to(DEV)
    pw = {"router": w["router"]}
    for e in range(E):
        pw.update({f"e{e}.{k}": w[f"{k}_{e}"] for k in ("gate", "up", "down")})
    if shared:
        pw.update({"shared.gate": w["shared_gate_proj"], "shared.up": w["shared_up"], "shared.down": w["shared_down"]})
    margins = []
    want = plain.mixture(x.cpu().double(), {k: v.cpu().double() for k, v in pw.items()}, "", m, margins)
    clear = margins[0] > 1e-4
    assert int(clear.sum()) >= T - 1
    for out32 in (False, True):
        got = RoutedExperts({**params, "out_dtype32": out32}, w, dtype).forward(x, step_ctx([T], [0], dtype=dtype))
        assert got.dtype == (torch.float32 if out32 else dtype)
        tol = dict(rtol=3e-2, atol=3e-2 * float(want.abs().max())) if dtype == torch.bfloat16 else dict(rtol=1e-4, atol=2e-5 * float(want.abs().max()))
        torch.testing.assert_close(got.cpu().double()[clear], want[clear], **tol)
