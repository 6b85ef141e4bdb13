"""The Tikizen design against its plain restatement (tests/plain_tikizen.py): the kernels of each mechanism alone, whole
models in every cutting of the requests, pages and slots that are used again, keys at the edges of a chunk and far away,
layers that read another layer's keys through a mask of their own, the first tokens of a sequence, long decoding through
chunks and pages, sizes that differ in everything, and greedy generation through the engine and its command lines."""
import json
import math
import os
import re
import subprocess
import sys

import numpy as np
import pytest
import torch

import plain_tikizen as plain
import traces
from tolerances import K, K_SELF, check_close

pytestmark = pytest.mark.gpu
DEV = "cuda:0"
ROOT = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))


def yarn(factor, original, fast=32.0, slow=1.0):
    return {"factor": factor, "original": original, "fast": fast, "slow": slow}


def _rot(rot):
    if rot is None:
        return {}
    r = {"base": rot[0], "dims": rot[1]}
    if len(rot) > 2:
        r["scaling"] = rot[2]
    return {"rot": r}


def dense(ff, limit=None):
    return {"kind": "dense", "ff": ff, **({"limit": limit} if limit is not None else {})}


def moe(experts, top, ff, shared=0):
    return {"kind": "moe", "expert": {"ff": ff}, "router": {"experts": experts, "top": top}, **({"shared": {"ff": shared}} if shared else {})}


def attn(heads, kv_heads, dim, vdim=None, scale=None, chunk=0, rot=None, kv_from=None, mlp=None):
    m = {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim or dim, "scale": scale if scale is not None else dim ** -0.5, **_rot(rot)}
    if chunk:
        m["mask"] = {"size": chunk}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def ret(heads, dim, vdim, decay, rot=None, mlp=None):
    return {"type": "retention", "mixer": {"heads": heads, "dim": dim, "vdim": vdim, "decay": list(decay), **_rot(rot)}, "mlp": mlp}


def mamba(heads, vdim, state, groups=1, norm_groups=1, conv=4, mlp=None):
    return {"type": "mamba2", "mixer": {"heads": heads, "vdim": vdim, "state": state, "groups": groups, "norm_groups": norm_groups, "conv": conv},
            "mlp": mlp}


def model_config(vocab, width, layers, eps=1e-5, alpha=1.0):
    return {"architecture": "Tikizen", "vocab": vocab, "width": width, "norm": {"eps": eps}, "postln_alpha": alpha, "layers": layers}


# A: every mixer and feed-forward; key and value widths differ both ways; a chunk shorter than two pages and one longer; a
# reader with the mask of the layer it reads; a layer without a feed-forward; several groups and norm groups
CONFIG_A = model_config(300, 96, [
    ret(3, 16, 24, (0.9, 0.99, 0.999), rot=(10000.0, 8), mlp=moe(7, 2, 40, 56)),
    mamba(4, 12, 16, groups=2, norm_groups=3, mlp=dense(80, 1.5)),
    attn(4, 2, 16, 24, chunk=21, rot=(5000.0, 16, yarn(4.0, 512)), mlp=moe(5, 3, 64, 24)),
    attn(8, 2, 16, 24, chunk=21, rot=(5000.0, 16, yarn(4.0, 512)), kv_from=2, mlp=dense(33, 0.7)),
    attn(4, 1, 24, 8, chunk=64, rot=(500.0, 8)),
], alpha=1.7)
# B: sizes that are multiples of nothing; as many key/value heads as heads; one expert of one; no limit, no shared expert,
# no rotation in one attention and one retention; convolutions of one tap and of five; a chunk of one position
CONFIG_B = model_config(211, 54, [
    mamba(3, 5, 7, conv=1, mlp=dense(21)),
    attn(3, 3, 10, 14, chunk=1, rot=(77.0, 4), mlp=moe(1, 1, 9)),
    ret(2, 5, 3, (1.0, 0.5), mlp=moe(6, 1, 13, 7)),
    mamba(2, 9, 11, groups=1, norm_groups=2, conv=5),
    attn(2, 1, 6, 6, chunk=50, scale=0.9, mlp=dense(17, 3.0)),
], eps=1e-6)
# C: heads of 64, 32, 96 and 128 (bfloat16 runs the tensor-core attention); widths that the tensor-core products take; a
# reader without a mask over a chunked layer's keys, a reader with a longer chunk, states of 64 and 128 rows
CONFIG_C = model_config(512, 128, [
    attn(4, 2, 64, 64, chunk=100, rot=(20000.0, 64, yarn(2.0, 1024)), mlp=dense(192, 2.5)),
    attn(8, 2, 64, 64, chunk=40, rot=(20000.0, 64, yarn(2.0, 1024)), kv_from=0, mlp=moe(16, 4, 64, 128)),
    mamba(4, 32, 64, groups=4, norm_groups=4, mlp=moe(9, 2, 96)),
    ret(2, 128, 64, (0.97, 0.995), rot=(10000.0, 64), mlp=dense(128, 4.0)),
    attn(2, 2, 96, 96, chunk=70, rot=(10000.0, 32), mlp=dense(64, 1.0)),
    attn(6, 2, 96, 96, rot=(10000.0, 32), kv_from=4),
    attn(2, 1, 128, 100, chunk=33),
], alpha=2.0)
# D: states and heads beyond the fast kernels' sizes; a head wider than 128; one group for all heads and as many as heads
CONFIG_D = model_config(157, 100, [
    ret(1, 136, 20, (0.98,), rot=(100.0, 136), mlp=moe(4, 4, 30, 50)),
    mamba(2, 40, 130, groups=2, norm_groups=1, conv=2, mlp=dense(60, 2.0)),
    attn(1, 1, 140, 16, chunk=45, rot=(10000.0, 20, yarn(3.0, 64, 8.0, 2.0))),
    mamba(6, 8, 24, groups=1, norm_groups=6, conv=3, mlp=moe(3, 2, 20)),
], alpha=1.3)
CONFIGS = {"a": CONFIG_A, "b": CONFIG_B, "c": CONFIG_C, "d": CONFIG_D}
LENGTHS = {"a": [1, 9, 40, 64, 131, 77, 2], "b": [3, 55, 150, 18, 97], "c": [200, 1, 65, 129, 30, 230], "d": [70, 2, 33, 140, 17]}
PAGE = {"a": 8, "b": 16, "c": 16, "d": 4}


def steer_routers(tensors, config, seed):
    """Gives every mixture `experts` coordinates of the stream: each token's embedding row is large and positive in `top` of
    them and negative in the others, the sublayers write little there, and the router reads them with a large weight beside
    its random ones. The choices then differ from token to token but none is close, so that a 16-bit rounding changes none."""
    rng = np.random.default_rng(seed)
    V, width, at = config["vocab"], config["width"], 0
    mixtures = [L["mlp"]["router"]["experts"] for L in config["layers"] if L.get("mlp") and L["mlp"]["kind"] == "moe"]
    total = sum(n for n in mixtures)
    assert total <= width // 2, "the routers' coordinates leave the stream too little room"
    for name, t in tensors.items():
        if total and name.endswith((".mix.o", ".down")):
            t[:total] *= 0.05
    for i, L in enumerate(config["layers"]):
        if not L.get("mlp") or L["mlp"]["kind"] != "moe":
            continue
        E, top = L["mlp"]["router"]["experts"], L["mlp"]["router"]["top"]
        r = tensors[f"l{i}.mlp.router"].float() * 0.2
        code = np.full((V, E), -1.0)
        for t in range(V):
            code[t, rng.permutation(E)[:top]] = 1.0
        code *= rng.uniform(0.8, 1.2, (V, E))
        std = float(tensors["embed"].float()[:, total:].std())
        tensors["embed"][:, at:at + E] = torch.tensor(2.5 * std * code).to(tensors["embed"].dtype)
        r[:, at:at + E] += 3.0 * torch.eye(E)
        at += E
        tensors[f"l{i}.mlp.router"] = r.to(tensors[f"l{i}.mlp.router"].dtype)
        tensors[f"l{i}.mlp.router.b"] *= 0.5


def write_model(folder, config, seed, dtype="bfloat16", init=None):
    from cellm_b200.weights import InitSpec, write_random_model
    from cellm_b200.weights.safetensors_io import SafetensorsFile, save_file
    init = init or InitSpec(linear_std=0.1, embedding_std=0.08, bias_std=0.3, norm_jitter=0.2)
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
    distance by which a chosen expert's sum lies above one left out."""
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
    d = tmp_path_factory.mktemp("tk")
    out = {}
    for i, (name, config) in enumerate(CONFIGS.items()):
        rng = np.random.default_rng(71 + i)
        reqs = {f"r{j}": rng.integers(0, config["vocab"], n).tolist() for j, n in enumerate(LENGTHS[name])}
        folder = write_model(d / name, config, 27 + i)
        cfg, w = load_plain(folder)
        out[name] = (folder, reqs, {rid: Ref(toks, cfg, w) for rid, toks in reqs.items()})
    return out


# Against the plain restatement in 64-bit. The recurrent state carries its 32-bit rounding from token to token and every
# read-out and stream is divided by its root mean square, so the 32-bit bound is 1e-5 of the logits' size; bfloat16 keeps
# the engine's bound, except for rows that rounding alone moves further.
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


def test_the_stream_after_every_layer(models):
    """The 32-bit stream after each layer against the plain model's."""
    from cellm_b200.parts import block as B
    from cellm_b200.replay import Replayer
    folder, reqs, _ = models["a"]
    cfg, w = load_plain(folder)
    toks = reqs["r3"]
    want = []
    plain.forward(toks, cfg, w, want)
    seen = []
    original = B.PostNormBlock.forward

    def recording(self, residual, ctx, cache):
        original(self, residual, ctx, cache)
        seen.append(residual.x.clone())
    B.PostNormBlock.forward = recording
    try:
        rp = Replayer(folder, "float32", 64, 8, 4, use_graphs=False)
        rp.step([{"id": "x", "tokens": toks, "want": [0]}], ["x"])
    finally:
        B.PostNormBlock.forward = original
    assert len(seen) == len(want) == 5
    for i, (x, ref) in enumerate(zip(seen, want)):
        check_close(x.cpu().numpy(), ref.numpy(), "float32", f"stream after layer {i}", k=KP["float32"])


def test_mixed_trace_reuses_pages_and_slots(models):
    folder, reqs, _ = models["a"]
    steps = traces.mixed(reqs)
    assert len(reqs) > 4                                     # more requests than state slots
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
def test_long_decoding_through_chunks_and_pages(models, name, dtype):
    """Most of the sequence decoded token by token: chunks begin and end among decoded tokens, pages of ended chunks are given
    back while the request lives, and the recurrent states walk a hundred and more single steps."""
    folder, reqs, ref = models[name]
    some = {rid: reqs[rid] for rid in (("r4", "r5") if name == "a" else ("r0", "r5"))}
    got = run_trace(folder, dtype, traces.tail_one_by_one(some, tail=190), 8)
    for rid, toks in some.items():
        against_plain(traces.as_matrix(got[rid], len(toks)), ref[rid], dtype, f"{name} {dtype} long tail {rid}")


def test_a_chunked_request_holds_its_chunk_only(tmp_path):
    """A request longer than the pools of its layers runs through: the pages of an ended chunk go back at once, in the pool
    that readers with two sizes of chunk share those behind the longer one, and the logits are the plain model's."""
    from cellm_b200.replay import Replayer
    rot = (100.0, 4)
    config = model_config(120, 48, [attn(2, 1, 8, chunk=20, rot=rot), attn(2, 1, 12, chunk=9, rot=rot), attn(4, 1, 12, chunk=24, rot=rot, kv_from=1),
                                    mamba(2, 6, 5)])
    folder = write_model(tmp_path / "w", config, 3)
    cfg, w = load_plain(folder)
    toks = np.random.default_rng(0).integers(0, 120, 210).tolist()
    ref = plain.forward(toks, cfg, w).numpy()
    rp = Replayer(folder, "float32", 64, 8, 4)               # 8 pages of 8 tokens a group: 64 keys for 210 tokens
    rows = []
    for i in range(0, len(toks), 5):
        part = toks[i:i + 5]
        rows.append(rp.step([{"id": "x", "tokens": part, "want": list(range(len(part)))}], []))
        n = i + len(part)
        for g, need in enumerate(rp.cache.paged_keys):
            assert (need.chunk, need.window) in ((20, 0), (0, 24))
            table = rp.cache.block_table(0, g, np.full((64,), -1, dtype=np.int32))
            first = n // 20 * 20 if need.chunk else n - 24 + 1
            assert [p >= 0 for p in table] == [(b + 1) * 8 > first for b in range(len(table))], (n, g)
    check_close(np.concatenate(rows), ref, "float32", "a request longer than its pools", k=KP["float32"])
    rp.step([], ["x"])
    assert rp.cache.live == 0 and all(rp.cache.free_pages(g) == rp.cache.group_pages[g] for g in range(len(rp.cache.group_pages)))


# ------------------------------------------------------------------------------------- chunk edges, far keys
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sharp_attention_at_the_edges_and_far_back(tmp_path, dtype):
    """A softmax so peaked (a large scale on queries and keys of unit root mean square) that a row's output is a few single
    keys wherever they lie: a key lost at a page border or at the start of a chunk, or one seen from the chunk before,
    changes the logits outright. The test first asserts, on the plain model, that such rows exist."""
    chunk = 45
    scale = 0.8 if dtype == "float32" else 0.4
    rot = (10000.0, 8)
    config = model_config(128, 64, [attn(4, 2, 16, scale=scale, chunk=chunk, rot=rot),
                                    attn(4, 2, 16, scale=scale, rot=rot, kv_from=0),
                                    attn(2, 1, 32, 16, scale=scale * 0.7, chunk=100, rot=(1000.0, 16, yarn(2.0, 256)))], alpha=1.0)
    from cellm_b200.weights import InitSpec
    folder = write_model(tmp_path / "sharp", config, 9, init=InitSpec(linear_std=0.25, embedding_std=0.1, bias_std=0.05, norm_jitter=0.1))
    cfg, w = load_plain(folder)
    rng = np.random.default_rng(4)
    toks = rng.integers(0, cfg["vocab"], 500).tolist()
    reqs = {"long": toks, "short": toks[:46]}
    ref = {rid: Ref(t, cfg, w, runs=4) for rid, t in reqs.items()}
    eps, pos = cfg["norm"]["eps"], torch.arange(len(toks))
    x0 = plain.rms(w["embed"][torch.tensor(toks)], eps) * w["embed.norm"]
    seen = []
    y, kept = plain.attention(x0, w, "l0.mix.", cfg["layers"][0]["mixer"], pos, eps, weights_out=seen)
    W = seen[0]                                                 # [heads, T, T]
    top, where = W[:, 100:].max(-1)
    assert float(top.median()) > (0.5 if dtype == "float32" else 0.25)
    rows = torch.arange(100, 500)[None]
    assert int((where == rows // chunk * chunk).sum()) >= 3      # the heaviest key is the first of the row's chunk
    full = torch.einsum("ihd,jhd->hij", plain.rms(plain.rotate_half((x0 @ w["l0.mix.q"].T).view(-1, 4, 16), pos, cfg["layers"][0]["mixer"]["rot"]), eps),
                        kept[0].repeat_interleave(2, dim=1)) * scale
    before = full[:, torch.arange(100, 500), (torch.arange(100, 500) // chunk * chunk - 1)]
    assert int((before > full[:, 100:].gather(2, where[..., None])[..., 0] + 1.0).sum()) >= 2      # the last key of the chunk before would win
    seen = []
    x1 = plain.rms(x0 + y, eps) * w["l0.norm1"]
    plain.attention(x1, w, "l1.mix.", cfg["layers"][1]["mixer"], pos, eps, kept, seen)
    top, where = seen[0][:, 400:].max(-1)
    assert float((torch.arange(400, 500)[None] - where).float().median()) > 40      # the reader reaches far back
    for fam in ("whole", "tail", "portions", "mixed"):
        for page in (8, 32):
            got = run_trace(folder, dtype, FAMILIES[fam](reqs), page)
            for rid, t in reqs.items():
                # so peaked a softmax passes a score's last bits on; a lost or surplus key moves a row by a tenth of the
                # logits' size and more
                against_plain(traces.as_matrix(got[rid], len(t)), ref[rid], dtype, f"sharp {dtype} {fam} page {page} {rid}", k32=1e-4)


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
def step_ctx(q_lens, ctx_lens, slots, tokens=None, dtype=torch.float32):
    """A step's index arrays for requests that bring q_lens[b] tokens after ctx_lens[b] earlier ones."""
    from cellm_b200.ops._state import error_word
    from cellm_b200.parts.base import StepContext
    i32 = lambda v: torch.tensor(v, dtype=torch.int32, device=DEV)
    T, B = sum(q_lens), len(q_lens)
    pos = [c + i for c, n in zip(ctx_lens, q_lens) for i in range(n)]
    seq = [b for b, n in enumerate(q_lens) for _ in range(n)]
    cu = [0] + list(np.cumsum(q_lens))
    return StepContext(T=T, B=B, dtype=dtype, device=torch.device(DEV), token_ids=i32(tokens if tokens is not None else [0] * T),
                       positions=i32(pos), seq_of_token=i32(seq), cu_seqlens=i32(cu), ctx_lens=i32(ctx_lens), slot_ids=i32(slots),
                       err=error_word(torch.device(DEV)), q_lens=list(q_lens), ctx_lens_host=list(ctx_lens), max_q_len=max(q_lens),
                       max_total_len=max(c + n for c, n in zip(ctx_lens, q_lens)))


def cuts_of(T, sizes):
    out, i, k = [], 0, 0
    while i < T:
        n = min(sizes[k % len(sizes)], T - i)
        out.append((i, n))
        i, k = i + n, k + 1
    return out


def walk_in_cuts(lens, slots, sizes, run):
    """Feeds sequences of `lens` side by side in portions of `sizes`; run(rows of each live sequence, ctx) -> [T, n]."""
    got = [[] for _ in lens]
    cuts = [cuts_of(L, sizes) for L in lens]
    for step in range(max(len(c) for c in cuts)):
        live = [b for b in range(len(lens)) if step < len(cuts[b])]
        ctx = step_ctx([cuts[b][step][1] for b in live], [cuts[b][step][0] for b in live], [slots[b] for b in live])
        rows = lambda src: torch.cat([src[b][cuts[b][step][0]:cuts[b][step][0] + cuts[b][step][1]] for b in live]).to(DEV).contiguous()
        o = run(rows, ctx).cpu()
        at = 0
        for b in live:
            got[b].append(o[at:at + cuts[b][step][1]])
            at += cuts[b][step][1]
    return [torch.cat(g) for g in got]


CUTTINGS = (("whole", (512,)), ("portions", (5, 1, 2, 11, 70)), ("single", (1,)))


@pytest.mark.parametrize("heads,groups,dim,vd", [(4, 2, 16, 12), (2, 1, 64, 64), (3, 3, 5, 7), (2, 2, 128, 40), (6, 3, 48, 48), (2, 1, 33, 9), (2, 1, 136, 20)])
@pytest.mark.parametrize("constants", [True, False])
def test_decay_walk_alone(heads, groups, dim, vd, constants):
    """Two sequences side by side in slots 3 and 1, fed whole and in portions down to one token: the walk with one decay and
    one writing factor per head (constants, or formed anew for every token) against the plain recurrence in 64-bit, the
    cuttings against each other bit for bit, other slots untouched. One head's decay is so near one that the first tokens
    still weigh at the end, another's so small that only the last token does."""
    from cellm_b200 import ops
    g = torch.Generator().manual_seed(heads * 100 + dim + constants)
    lens, slots, n = [201, 19], [3, 1], groups * dim
    ld = 2 * n + heads * vd + 4                                            # q | k | v and something behind them
    proj = [torch.randn(L, ld, generator=g) for L in lens]
    if constants:
        d0 = torch.rand(heads, generator=g) * 0.3 + 0.65
        d0[0], d0[-1] = 0.9995, 0.01
        w0 = torch.rand(heads, generator=g) + 0.2
        decay, write = [d0.expand(L, heads) for L in lens], [w0.expand(L, heads) for L in lens]
    else:
        decay = [torch.rand(L, heads, generator=g) * 0.5 + 0.5 for L in lens]
        for d in decay:
            d[:, 0] = 0.9995
        write = [torch.rand(L, heads, generator=g) * 2 for L in lens]
    want = []
    for b, L in enumerate(lens):
        p = proj[b].double()
        q, k = (p[:, i * n:(i + 1) * n].reshape(L, groups, dim).repeat_interleave(heads // groups, dim=1) for i in range(2))
        want.append(plain.decayed_sums(q, k, p[:, 2 * n:2 * n + heads * vd].reshape(L, heads, vd), decay[b].double(), write[b].double()).reshape(L, -1))
    outs = {}
    for name, sizes in CUTTINGS:
        state = torch.full((4, heads, dim, vd), 7.0, device=DEV)
        state[slots] = 0

        def run(rows, ctx):
            p = rows(proj)
            d, wr = (d0.to(DEV), w0.to(DEV)) if constants else (rows(decay), rows(write))
            return ops.decay_scan(p, p[:, n:], p[:, 2 * n:], d, wr, state, ctx, heads, groups, dim, vd)
        outs[name] = walk_in_cuts(lens, slots, sizes, run)
        assert float(state[0].min()) == 7.0 and float(state[2].max()) == 7.0
        for b in range(len(lens)):
            torch.testing.assert_close(outs[name][b].double(), want[b], rtol=3e-5, atol=3e-5 * float(want[b].abs().max()))
    for b in range(len(lens)):
        assert torch.equal(outs["whole"][b], outs["portions"][b]) and torch.equal(outs["whole"][b], outs["single"][b])
    # long portions in chunks on the tensor cores, the others token by token, and both kinds side by side
    log = lambda d: torch.log(d.clamp_min(1e-30))
    for sizes in ((512,), (64, 65, 12), (70, 1), (63, 100)):
        state = torch.full((4, heads, dim, vd), 7.0, device=DEV)
        state[slots] = 0

        def run_chunks(rows, ctx):
            p = rows(proj)
            d, wr = (d0.to(DEV), w0.to(DEV)) if constants else (rows(decay), rows(write))
            return ops.decay_scan(p, p[:, n:], p[:, 2 * n:], d, wr, state, ctx, heads, groups, dim, vd, log(d).contiguous())
        got = walk_in_cuts(lens, slots, sizes, run_chunks)
        assert float(state[0].min()) == 7.0 and float(state[2].max()) == 7.0
        for b in range(len(lens)):
            torch.testing.assert_close(got[b].double(), want[b], rtol=1e-4, atol=1e-4 * float(want[b].abs().max()))
    # no writing factor: one
    state = torch.zeros((1, heads, dim, vd), device=DEV)
    p = proj[1].to(DEV)
    a = ops.decay_scan(p, p[:, n:], p[:, 2 * n:], decay[1][0].contiguous().to(DEV), None, state, step_ctx([19], [0], [0]), heads, groups, dim, vd)
    state.zero_()
    b = ops.decay_scan(p, p[:, n:], p[:, 2 * n:], decay[1][0].contiguous().to(DEV), torch.ones(heads, device=DEV), state, step_ctx([19], [0], [0]), heads,
                       groups, dim, vd)
    assert torch.equal(a, b)


def part_in_cuts(kind, params, weights, x, sizes, needs):
    """A mixer part alone in 32-bit over sequences x[b], its state in slots of its own."""
    from cellm_b200.parts.base import CacheBinding
    from cellm_b200.parts.registry import part_class
    part = part_class("mixer", kind)(params, {k: v.to(DEV) for k, v in weights.items()}, torch.float32)
    states = tuple(CacheBinding(need=n, state=torch.zeros((4,) + tuple(n.shape), device=DEV), num_slots=4) for n in needs)
    cache = states[0] if len(states) == 1 else CacheBinding(need=needs, parts=states)
    return walk_in_cuts([len(t) for t in x], [2, 0], sizes, lambda rows, ctx: part.forward(rows(x), ctx, cache))


@pytest.mark.parametrize("H,heads,dim,vd,rot", [(40, 3, 8, 6, (100.0, 4)), (64, 2, 64, 32, (10000.0, 64)), (33, 1, 5, 9, None),
                                                 (48, 4, 16, 16, (50.0, 16, yarn(8.0, 32, 4.0, 1.0)))])
def test_retention_alone(H, heads, dim, vd, rot):
    from cellm_b200.config.plan import PartSpec
    from cellm_b200.parts.base import FixedState
    g = torch.Generator().manual_seed(H + dim)
    rnd = lambda *s: torch.randn(*s, generator=g)
    w = {"q": rnd(heads * dim, H) / H ** 0.5, "k": rnd(heads * dim, H) / H ** 0.5, "v": rnd(heads * vd, H) / H ** 0.5, "g": rnd(heads * vd, H) / H ** 0.5,
         "o": rnd(H, heads * vd) / (heads * vd) ** 0.5}
    decay = [0.999, 0.9, 0.5, 0.97][:heads]
    m = {"heads": heads, "dim": dim, "vdim": vd, "decay": decay, **_rot(rot)}
    pos = None if rot is None else PartSpec("rope", {"head_dim": dim, "rotary_dim": rot[1], "theta": rot[0], "layout": "half",
                                                     "scaling": rot[2] if len(rot) > 2 else None})
    params = {"hidden_size": H, "heads": heads, "dim": dim, "value_dim": vd, "decay": decay, "eps": 1e-5, "position": pos, "out_dtype32": True}
    x = [rnd(90, H), rnd(31, H)]
    want = [plain.retention(t.double(), {k: v.double() for k, v in w.items()}, "", m, torch.arange(len(t)), 1e-5) for t in x]
    outs = {name: part_in_cuts("retention", params, w, x, sizes, (FixedState((heads, dim, vd)),)) for name, sizes in CUTTINGS}
    for name in outs:
        for b in range(2):
            torch.testing.assert_close(outs[name][b].double(), want[b], rtol=2e-4, atol=2e-5 * float(want[b].abs().max()))


@pytest.mark.parametrize("H,heads,vd,n,groups,ng,taps", [(40, 4, 6, 8, 2, 3, 4), (64, 2, 32, 64, 1, 1, 4), (33, 3, 5, 7, 3, 5, 1), (48, 2, 16, 16, 1, 2, 2),
                                                          (48, 2, 16, 16, 2, 4, 3), (32, 1, 8, 130, 1, 1, 6)])
def test_mamba2_alone(H, heads, vd, n, groups, ng, taps):
    """Convolutions of one to six taps whose past lies in the portion, in the state or before the start; step sizes on both
    sides of softplus' bend; several groups of B and C, parts of the norm that do not end where a head ends."""
    from cellm_b200.parts.base import FixedState
    g = torch.Generator().manual_seed(H + n + taps)
    rnd = lambda *s: torch.randn(*s, generator=g)
    inner, C = heads * vd, heads * vd + 2 * groups * n
    w = {"in": rnd(inner + C + heads, H) / H ** 0.5, "conv": rnd(C, taps) * 0.6, "conv_bias": rnd(C) * 0.3, "dt_bias": rnd(heads) * 3, "A_log": rnd(heads),
         "D": rnd(heads), "norm": 1 + 0.3 * rnd(inner), "o": rnd(H, inner) / inner ** 0.5}
    m = {"heads": heads, "vdim": vd, "state": n, "groups": groups, "norm_groups": ng}
    pw = {("conv.b" if k == "conv_bias" else k): v.double() for k, v in w.items()}
    params = {"hidden_size": H, "heads": heads, "value_dim": vd, "state": n, "groups": groups, "norm_groups": ng, "conv_taps": taps, "eps": 1e-5,
              "out_dtype32": True}
    x = [rnd(600, H), rnd(31, H)]           # 600: the preparation walks runs of tokens
    want = [plain.mamba2(t.double(), pw, "", m, 1e-5) for t in x]
    needs = ((FixedState((taps - 1, C)),) if taps > 1 else ()) + (FixedState((heads, n, vd)),)
    for name, sizes in (("whole", (1024,)), ("portions", (5, 1, 2, 11, 300)), ("pairs", (2,))):
        outs = part_in_cuts("mamba2", params, w, x, sizes, needs)
        for b in range(2):
            torch.testing.assert_close(outs[b].double(), want[b], rtol=3e-4, atol=3e-5 * float(want[b].abs().max()))


class _Pages:
    """A pool of keys and values with one request's pages in an order of their own."""
    def __init__(self, n_tokens, nkv, hd, vd, page, dtype, g):
        n_pages = -(-n_tokens // page) + 3
        self.k = torch.zeros(n_pages, nkv, page, hd, dtype=dtype, device=DEV)
        self.v = torch.zeros(n_pages, nkv, page, vd, dtype=dtype, device=DEV)
        order = torch.randperm(n_pages, generator=g)[: -(-n_tokens // page)]
        self.block_table = order.to(torch.int32).reshape(1, -1).to(DEV)
        self.page_size, self.order = page, order

    def put(self, keys, vals):
        for j in range(keys.shape[0]):
            p, s = int(self.order[j // self.page_size]), j % self.page_size
            self.k[p, :, s] = keys[j].to(self.k.dtype)
            self.v[p, :, s] = vals[j].to(self.v.dtype)


@pytest.mark.parametrize("nh,nkv,hd,vd,rot,norm,width", [(4, 2, 16, 24, (10000.0, 8), True, 32), (3, 1, 10, 6, None, True, 10), (2, 2, 96, 96, (500.0, 96, yarn(4.0, 64)), True, 96),
                                                          (1, 1, 140, 16, (100.0, 20, yarn(3.0, 64, 8.0, 2.0)), True, 140), (8, 4, 64, 64, (1e6, 64), False, 64)])
def test_turned_and_normed_heads_alone(nh, nkv, hd, vd, rot, norm, width):
    """Rotation (part of a head or all of it, stretched by place with its amplitude), then the norm over all of a head's
    entries; queries into a dense buffer, keys and values into pages, zeros behind a widened head's entries; and the same
    queries where the layer has none of its own keys."""
    from cellm_b200 import ops
    from cellm_b200.parts.rope import RotaryEmbedding
    g = torch.Generator().manual_seed(nh * 7 + hd)
    T, page, eps, start = 37, 8, 1e-5, 5000
    width_v = width if width != hd or hd == vd else vd
    pos_part = RotaryEmbedding({"head_dim": hd, "rotary_dim": rot[1], "theta": rot[0], "layout": "half", "scaling": rot[2] if len(rot) > 2 else None},
                               DEV) if rot else None
    proj = torch.randn(T, nh * hd + nkv * (hd + vd), generator=g)
    pool = _Pages(start + T, nkv, width, width_v, page, torch.float32, g)
    pool.k += 9.0
    ctx = step_ctx([T], [start], [0])
    freq, n_rot, amp = (pos_part.inv_freq, rot[1], pos_part.amplitude) if rot else (None, 0, 1.0)
    q = ops.turned_attn_prep(proj.to(DEV), freq, n_rot, False, amp, eps if norm else None, ctx, pool, nh, nkv, hd, vd, width, torch.float32)
    positions = torch.arange(start, start + T)
    p = proj.double()
    r = _rot(rot).get("rot")
    turn = lambda x: plain.rotate_half(x, positions, r)
    unit = (lambda x: plain.rms(x, eps)) if norm else (lambda x: x)
    want_q, want_k = unit(turn(p[:, :nh * hd].reshape(T, nh, hd))), unit(turn(p[:, nh * hd:(nh + nkv) * hd].reshape(T, nkv, hd)))
    want_v = p[:, (nh + nkv) * hd:].reshape(T, nkv, vd)
    q = q.cpu().double().reshape(T, nh, width)
    torch.testing.assert_close(q[..., :hd], want_q, rtol=1e-5, atol=2e-5)
    assert not q[..., hd:].any()
    for t in (0, 1, page - 1, page, T - 1):
        j = start + t
        pg, s = int(pool.order[j // page]), j % page
        k, v = pool.k[pg, :, s].cpu().double(), pool.v[pg, :, s].cpu().double()
        torch.testing.assert_close(k[:, :hd], want_k[t], rtol=1e-5, atol=2e-5)
        torch.testing.assert_close(v[:, :vd], want_v[t], rtol=1e-6, atol=1e-6)
        assert not k[:, hd:].any() and not v[:, vd:].any()
    assert float(pool.k[int(pool.order[0])].min()) == 9.0                     # other tokens' rows stay
    only = ops.turned_attn_prep(proj[:, :nh * hd].contiguous().to(DEV), freq, n_rot, False, amp, eps if norm else None, ctx, pool, nh, 0, hd, vd, width,
                                torch.float32)
    assert torch.equal(only.cpu().double().reshape(T, nh, width), q)


def test_stretched_frequencies_against_plain():
    from cellm_b200.parts.rope import RotaryEmbedding
    for base, dims, sc in ((300000.0, 80, yarn(3.0, 4096)), (10000.0, 64, yarn(16.0, 4096, 32.0, 1.0)), (100.0, 20, yarn(3.0, 64, 8.0, 2.0)),
                           (1e6, 8, yarn(1.0, 100)), (10000.0, 16, yarn(4.0, 1e9)), (10000.0, 16, yarn(4.0, 1.0)), (50.0, 2, yarn(5.0, 200, 4.0, 4.0))):
        part = RotaryEmbedding({"head_dim": dims, "rotary_dim": dims, "theta": base, "scaling": sc}, "cpu")
        f, amp = plain.frequencies({"base": base, "dims": dims, "scaling": sc})
        torch.testing.assert_close(part.inv_freq.double().sum(1), f, rtol=1e-12, atol=0)
        assert part.amplitude == pytest.approx(amp, abs=1e-15)


@pytest.mark.parametrize("chunk,page", [(16, 8), (21, 8), (33, 16), (1, 4), (0, 8), (130, 32), (400, 16), (64, 64)])
def test_chunked_attention_sees_exactly_its_chunk(chunk, page):
    """One key at a time carries a value that stands out; a query scores every key alike. The output tells which keys the row
    summed: those of its own run of positions up to itself, none of the run before. Prompt rows and single decoded rows, the
    first and last of a chunk and keys at page borders included; the plain kernel and, for the number of keys, the
    tensor-core one."""
    from cellm_b200 import ops
    g = torch.Generator().manual_seed(chunk * 100 + page)
    T, nh, nkv = 150, 2, 1
    for dtype, hd, vd in ((torch.float32, 8, 6), (torch.bfloat16, 32, 32), (torch.bfloat16, 96, 96)):
        keys = torch.zeros(T, nkv, hd)
        keys[:, :, 0] = 1.0
        vals = torch.zeros(T, nkv, vd)
        j = torch.arange(T)
        vals[:, 0, 0], vals[:, 0, 1], vals[:, 0, 2] = j % 8, (j // 8) % 8, j // 64      # a key's number, in digits bfloat16 holds exactly
        pool = _Pages(T, nkv, hd, vd, page, dtype, g)
        pool.put(keys, vals)
        q = torch.zeros(T, nh, hd)
        q[:, :, 0] = 0.5
        edges = [0, T - 1, page - 1, page, chunk - 1, chunk, chunk + 1, 2 * chunk - 1, 2 * chunk]
        for rows in [list(range(T))] + [[r] for r in edges]:
            rows = [r for r in rows if 0 <= r < T]
            if not rows:
                continue
            ctx = step_ctx([T], [0], [0]) if len(rows) == T else step_ctx([1], [rows[0]], [0])
            qq = q[rows].reshape(len(rows), -1).to(dtype).to(DEV).contiguous()
            # pages of keys before the row's chunk are given back in the engine: nothing may read them
            table = pool.block_table.clone()
            if len(rows) == 1 and chunk:
                pool.block_table[0, :rows[0] // chunk * chunk // page] = -1
            if dtype == torch.float32:
                out = ops.attention_plain_chunked(qq, pool, ctx, nh, nkv, hd, vd, 1.0, chunk)
            else:
                out = ops.attention_flash_chunked(qq, pool, ctx, nh, nkv, hd, 1.0, chunk)
            pool.block_table.copy_(table)
            out = out.cpu().double().reshape(len(rows), nh, vd)
            assert int(ctx.err.item()) == 0
            tol = 1e-4 if dtype == torch.float32 else 6e-3
            for n, i in enumerate(rows):
                seen = torch.tensor([k for k in range(i + 1) if chunk == 0 or k // chunk == i // chunk])
                for c, digit in enumerate((seen % 8, (seen // 8) % 8, seen // 64)):
                    mean = float(digit.double().mean())
                    assert abs(float(out[n, 1, c]) - mean) <= tol * (1 + mean), (dtype, i, c)


@pytest.mark.parametrize("hd,vd,chunk", [(64, 64, 50), (32, 32, 0), (128, 128, 7), (96, 96, 33), (96, 80, 200), (40, 24, 64), (64, 64, 300), (16, 16, 21)])
def test_tensor_core_attention_against_the_plain_kernel(tmp_path, hd, vd, chunk):
    """The bfloat16 mixer on the paged mma.sync attention against the plain kernel on the same cache, for a prompt, portions
    and single tokens (chunks of 200 and more: a single token's keys are cut into pieces), heads widened with zeros included."""
    from cellm_b200.parts import turned_attention as TA
    config = model_config(64, 64, [attn(4, 2, hd, vd, chunk=chunk, rot=(10000.0, hd // 2)), attn(4, 2, hd, vd, rot=(10000.0, hd // 2), kv_from=0)])
    folder = write_model(tmp_path / "t", config, 5)
    toks = np.random.default_rng(1).integers(0, 64, 300).tolist()
    reqs = {"x": toks, "y": toks[:33]}
    outs = {}
    for tc in (True, False):
        TA.OPTIONS["tensor_cores"] = tc
        try:
            outs[tc] = {fam: run_trace(folder, "bfloat16", FAMILIES[fam](reqs), 16) for fam in ("whole", "tail", "portions")}
        finally:
            TA.OPTIONS["tensor_cores"] = True
    for fam in outs[True]:
        for rid, t in reqs.items():
            check_close(traces.as_matrix(outs[True][fam][rid], len(t)), traces.as_matrix(outs[False][fam][rid], len(t)), "bfloat16",
                        f"tensor cores vs plain, {fam} {rid}", k=K_SELF["bfloat16"])


def test_tcgen05_attention_in_chunks_against_the_mma_kernel(tmp_path):
    """Prompt portions that fill its tiles run the attention of heads of 64 on tcgen05 (scores and outputs in tensor memory):
    chunks that end inside a tile of rows, at its edge and beyond the prompt, a reader with a chunk of its own, portions
    that start inside a chunk; against the plain model and the mma.sync kernel on the same requests."""
    from cellm_b200 import ops
    from cellm_b200.parts import turned_attention as TA
    from cellm_b200.runtime import program
    rot = (10000.0, 32)
    config = model_config(80, 128, [attn(8, 2, 64, chunk=70, rot=rot, mlp=dense(64, 2.0)), attn(16, 2, 64, chunk=32, rot=rot, kv_from=0),
                                    attn(4, 1, 64, chunk=256, rot=rot, mlp=moe(4, 2, 64, 64)), attn(4, 4, 64, rot=rot)], alpha=1.5)
    folder = write_model(tmp_path / "t", config, 8)
    cfg, w = load_plain(folder)
    toks = np.random.default_rng(2).integers(0, 80, 700).tolist()
    reqs = {"x": toks, "y": toks[100:333]}
    ref = {rid: Ref(t, cfg, w) for rid, t in reqs.items()}
    calls = []
    original = ops.attention_tc_chunked

    def counting(*a, **k):
        calls.append(1)
        return original(*a, **k)
    ops.attention_tc_chunked = counting
    old = program.OPTIONS["attention_tc_min_ctas"]
    program.OPTIONS["attention_tc_min_ctas"] = 1
    outs = {}
    try:
        for on in (True, False):
            TA.OPTIONS["tcgen05"] = on
            n = len(calls)
            outs[on] = {fam: run_trace(folder, "bfloat16", make(reqs), 16) for fam, make in
                        (("whole", traces.whole), ("portions", lambda r: traces.portions(r, (300, 64, 130, 2))))}
            assert (len(calls) > n) == on
    finally:
        TA.OPTIONS["tcgen05"] = True
        program.OPTIONS["attention_tc_min_ctas"] = old
        ops.attention_tc_chunked = original
    for fam in outs[True]:
        for rid, t in reqs.items():
            against_plain(traces.as_matrix(outs[True][fam][rid], len(t)), ref[rid], "bfloat16", f"tcgen05 {fam} {rid}")
            check_close(traces.as_matrix(outs[True][fam][rid], len(t)), traces.as_matrix(outs[False][fam][rid], len(t)), "bfloat16",
                        f"tcgen05 vs mma.sync, {fam} {rid}", k=K_SELF["bfloat16"])


@pytest.mark.parametrize("T,H", [(9, 54), (5, 56), (3, 2048), (70, 1100), (2, 4096), (2, 8192), (2, 9000), (4, 512)])
def test_norm_behind_the_sum_and_normed_embedding(T, H):
    from cellm_b200 import ops
    g = torch.Generator().manual_seed(T * 7 + H)
    rnd = lambda *s: torch.randn(*s, generator=g)
    x, a, w = rnd(T, H) * 3 + 0.5, rnd(T, H), 1 + 0.2 * rnd(H)
    for add_dtype, act in ((torch.float32, torch.float32), (torch.float32, torch.bfloat16), (torch.bfloat16, torch.bfloat16)):
        ad = a.to(add_dtype)
        want = plain.rms(1.7 * x.double() + ad.double(), 1e-5) * w.double()
        xd = x.to(DEV).clone()
        y = ops.post_norm(xd, ad.to(DEV), 1.7, w.to(DEV), 1e-5, act)
        torch.testing.assert_close(xd.cpu().double(), want, rtol=1e-5, atol=1e-5)
        assert torch.equal(y, xd.to(act))
    err = torch.zeros(1, dtype=torch.int32, device=DEV)
    ids = torch.randint(0, 23, (T,), generator=g)
    for dtype in (torch.float32, torch.bfloat16):
        table = (rnd(23, H) * 0.05).to(dtype)
        got = ops.embed_norm(table.to(DEV), ids.to(torch.int32).to(DEV), w.to(DEV), 1e-3, err, 2.0)
        torch.testing.assert_close(got.cpu().double(), plain.rms(2.0 * table.double()[ids], 1e-3) * w.double(), rtol=1e-5, atol=1e-5)
    assert int(err.item()) == 0
    ops.embed_norm(table.to(DEV), torch.full((T,), 23, dtype=torch.int32, device=DEV), w.to(DEV), 1e-3, err)
    assert int(err.item()) == 1


@pytest.mark.parametrize("limit", [0.8, None])
@pytest.mark.parametrize("T,H,ff", [(1, 64, 128), (5, 64, 80), (40, 128, 200), (64, 256, 1000), (100, 128, 192), (300, 64, 640), (700, 2048, 512), (3, 54, 33),
                                    (200, 54, 21), (9, 2048, 8192)])
def test_clamped_gate_alone(T, H, ff, limit):
    """The feed-forward part in both element types: gates and ups on both sides of the limits; bfloat16 joins them in the
    product's epilogue (swapped tiles with and without a split of K, plain tiles, the persistent kernel, widths that are no
    multiple of 64), other widths in a kernel of its own."""
    from cellm_b200.parts.gated_mlp import GatedMLP
    if ff * H > 1 << 23 and limit is None:
        pytest.skip("the largest shape once")
    g = torch.Generator().manual_seed(T + H + ff)
    for dtype in (torch.float32, torch.bfloat16):
        w = {"gate": torch.randn(ff, H, generator=g) * 1.5 / H ** 0.5, "up": torch.randn(ff, H, generator=g) * 1.5 / H ** 0.5,
             "down": torch.randn(H, ff, generator=g) / ff ** 0.5}
        w = {k: v.to(dtype).to(DEV) for k, v in w.items()}
        x = torch.randn(T, H, generator=g).to(dtype).to(DEV)
        pw = {k: v.cpu().double() for k, v in w.items()}
        want = plain.dense(x.cpu().double(), pw, "", limit)
        part = GatedMLP({"hidden_size": H, "ff_dim": ff, "activation": "clamped", "limit": limit, "slope": 1.702, "out_dtype32": True}, w, dtype)
        assert part.fused == (dtype == torch.bfloat16 and H % 8 == 0)
        got = part.forward(x, step_ctx([T], [0], [0], dtype=dtype))
        assert got.dtype == torch.float32
        k = 1e-2 if dtype == torch.bfloat16 else 1e-5
        torch.testing.assert_close(got.cpu().double(), want, rtol=k, atol=k * float(want.abs().max()))


MIXTURES = [  # H, experts, top, ff, shared ff
    (96, 12, 4, 40, 56), (54, 5, 4, 21, 33), (128, 16, 1, 64, 0), (64, 8, 8, 32, 16), (2048, 64, 6, 256, 512), (104, 6, 2, 24, 8), (256, 32, 3, 128, 0),
    (64, 1, 1, 70, 20), (64, 4, 4, 4096, 0), (72, 3, 2, 192, 128),
]


@pytest.mark.parametrize("T", [1, 5, 16, 17, 150, 300])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("H,E,top,ff,sff", MIXTURES)
def test_gated_experts_against_plain(dtype, T, H, E, top, ff, sff):
    """The part alone on random inputs: the plain function reads the same (rounded) input and weights, so every choice is the
    same one unless two sums lie within 32-bit rounding of each other. Few tokens take the row-by-row kernels, many (under
    bfloat16, with widths the tensor cores take) the grouped products."""
    from cellm_b200.parts.routed_experts import RoutedExperts
    if (H == 2048 or ff == 4096) and T not in (5, 150):
        pytest.skip("the large shapes at two sizes")
    g = torch.Generator().manual_seed(H * 7 + E)
    rnd = lambda *s: torch.randn(*s, generator=g)
    w = {"router": rnd(E, H) * 3 / H ** 0.5, "correction": rnd(E) * 0.7}
    for e in range(E):
        w[f"gate_{e}"], w[f"up_{e}"], w[f"down_{e}"] = rnd(ff, H) / H ** 0.5, rnd(ff, H) / H ** 0.5, rnd(H, ff) / ff ** 0.5
    if sff:
        w.update(shared_gate_proj=rnd(sff, H) / H ** 0.5, shared_up=rnd(sff, H) / H ** 0.5, shared_down=rnd(H, sff) / sff ** 0.5, shared_gate=rnd(1, H) / H ** 0.5)
    w = {k: v.to(dtype).to(DEV) for k, v in w.items()}
    part = RoutedExperts({"hidden_size": H, "experts": E, "top": top, "ff_dim": ff, "activation": "silu", "scores": "softmax", "gated": True,
                          "shared_ff": sff, "out_dtype32": True}, w, dtype)
    x = rnd(T, H).to(dtype).to(DEV)
    got = part.forward(x, step_ctx([T], [0], [0], dtype=dtype))
    assert got.dtype == torch.float32
    pw = {"router": w["router"], "router.b": w["correction"]}
    for e in range(E):
        pw.update({f"e{e}.{k}": w[f"{k}_{e}"] for k in ("gate", "up", "down")})
    if sff:
        pw.update({"shared.gate": w["shared_gate_proj"], "shared.up": w["shared_up"], "shared.down": w["shared_down"], "shared.sg": w["shared_gate"]})
    want = plain.mixture(x.cpu().double(), {k: v.cpu().double() for k, v in pw.items()}, "",
                         {"router": {"experts": E, "top": top}, "shared": {"ff": sff} if sff else None})
    tol = dict(rtol=3e-2, atol=3e-2 * float(want.abs().max())) if dtype == torch.bfloat16 else dict(rtol=1e-4, atol=2e-5 * float(want.abs().max()))
    torch.testing.assert_close(got.cpu().double(), want, **tol)


def test_softmax_choice_and_weights():
    """The router alone against the plain choice: ties go to the lower index, the bias takes part in choice and weight, sums
    far from zero do not overflow, and no bias at all."""
    from cellm_b200.ops._lib import fn, ptr, stream_of, tag
    g = torch.Generator().manual_seed(2)
    for E, top in ((8, 3), (6, 1), (12, 5), (1, 1), (64, 6), (5, 5)):
        T = 40
        z = torch.randn(T, E + 1, generator=g) * 2
        z[3, :E] = 0.0
        z[4, :E] += 300.0
        z[5, :E] -= 300.0
        bias = torch.randn(E, generator=g)
        if E > 1:
            bias[1] = bias[0]
        for b, dtype in ((bias, torch.float32), (bias.to(torch.bfloat16), torch.bfloat16), (None, torch.float32)):
            idx = torch.empty(T, top, dtype=torch.int32, device=DEV)
            wts, gate = torch.empty(T, top, device=DEV), torch.empty(T, device=DEV)
            zd, bd = z.to(DEV), None if b is None else b.to(DEV)
            assert fn("kernels_common", "cellm_route_softmax")(ptr(idx), ptr(wts), ptr(gate), ptr(zd), E + 1, ptr(bd), tag(dtype), T, E, top, 1.0, 1,
                                                               stream_of(zd)) == 0
            s = z[:, :E] + (b.float() if b is not None else 0.0)           # the sums as 32-bit numbers: ties stay ties
            want_idx, want_w = plain.choose(s.double(), top)
            assert torch.equal(idx.cpu().long(), want_idx), (E, top)
            torch.testing.assert_close(wts.cpu().double(), want_w, rtol=1e-5, atol=1e-6)
            torch.testing.assert_close(gate.cpu().double(), torch.sigmoid(z[:, E].double()), rtol=1e-5, atol=1e-7)


@pytest.mark.parametrize("T,heads,vd,groups", [(5, 4, 12, 3), (3, 2, 64, 1), (70, 3, 7, 7), (2, 64, 64, 8)])
def test_norms_behind_the_recurrences(T, heads, vd, groups):
    from cellm_b200 import ops
    g = torch.Generator().manual_seed(T + heads)
    rnd = lambda *s: torch.randn(*s, generator=g)
    inner = heads * vd
    o, x, z, D, w = rnd(T, inner), rnd(T, inner + 5), rnd(T, inner + 3) * 2, rnd(heads), 1 + 0.2 * rnd(inner)
    for act, k in ((torch.float32, 1e-5), (torch.bfloat16, 8e-3)):
        got = ops.gated_group_norm(o.to(DEV), x.to(DEV), D.to(DEV), z.to(DEV), w.to(DEV), vd, groups, 1e-5, act).cpu().double()
        v = (o.double() + D.double().repeat_interleave(vd) * x.double()[:, :inner]) * plain.silu(z.double()[:, :inner])
        torch.testing.assert_close(got, plain.rms(v.view(T, groups, -1), 1e-5).reshape(T, inner) * w.double(), rtol=k, atol=k)
        got = ops.head_norm_silu(o.to(DEV), z.to(DEV)[:, 3:], heads, vd, 1e-5, act).cpu().double()
        want = plain.rms(o.double().view(T, heads, vd), 1e-5).reshape(T, inner) * plain.silu(z.double()[:, 3:])
        torch.testing.assert_close(got, want, rtol=k, atol=k)
