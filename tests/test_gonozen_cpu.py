"""What the Gonozen design adds that needs no GPU: its configuration reader (what the file leaves out does not exist; faults name
their key), the plan and the tensors it expects, what the layers keep in the cache, which kernels a step launches and with
which sizes, how a result's norm meets the next norm or anything else that needs the stream, and what the parts refuse."""
import copy

import pytest
import torch

from cellm_b200 import models, parts  # noqa: F401  (register architectures and parts)
from cellm_b200.config import ConfigError, config_from_dict
from cellm_b200.parts import PagedKV
from cellm_b200.weights.loader import expected_tensors
from launch_recorder import Recorder, run_step, zero_model

ROT = {"base": 100.0, "dims": 16, "scaling": {"factor": 2.0, "original": 64, "fast": 8.0, "slow": 1.0}}
MOE = {"kind": "moe", "expert": {"ff": 40, "limit": 0.75}, "router": {"experts": 12, "top": 3, "groups": {"count": 4, "keep": 2}}, "shared": {"ff": 70, "limit": 1.25}}
LAT = {"type": "latent_attention", "mixer": {"heads": 4, "dim": 32, "rot_dim": 16, "vdim": 24, "kv_rank": 64, "scale": 0.3, "rot": ROT}, "mlp": MOE}
WIN = {"type": "latent_attention_2", "mixer": {"heads": 2, "dim": 48, "vdim": 40, "kv_rank": 64, "q_rank": 56, "scale": 0.2, "mask": {"size": 9}}, "mlp": MOE}


def config(layers=(LAT, WIN), **top):
    return copy.deepcopy({"architecture": "Gonozen", "vocab": 90, "width": 128, "norm": {"eps": 1e-4}, "logit_softcap": 21.0, "layers": list(layers), **top})


def without(layer, *keys):
    layer = copy.deepcopy(layer)
    for k in keys:
        at = layer
        *path, last = k.split(".")
        for p in path:
            at = at[p]
        at.pop(last)
    return layer


def test_the_reader_takes_every_constant_from_the_file():
    cfg, plan = config_from_dict(config())
    assert (cfg.vocab, cfg.width, cfg.norm_eps, cfg.logit_softcap) == (90, 128, 1e-4, 21.0)
    a, b = plan.layers
    assert (a.mixer.params["gate"], a.mixer.params["rot_dim"], a.mixer.params["scale"]) == (True, 16, 0.3)
    assert a.mixer.params["position"].params == {"head_dim": 16, "rotary_dim": 16, "theta": 100.0, "layout": "half", "scaling": ROT["scaling"]}
    assert (b.mixer.params["q_rank"], b.mixer.params["window"], b.mixer.params["sinks"], b.mixer.params["rot_dim"]) == (56, 9, True, 0)
    ff = a.feed_forward.params
    assert (ff["experts"], ff["top"], ff["ff_dim"], ff["groups"], ff["keep_groups"], ff["scores"], ff["activation"]) == (12, 3, 40, 4, 2, "softmax_all", "clamped")
    assert (ff["limit"], ff["shared_limit"], ff["shared_ff"], ff["slope"], ff["shared_gate"]) == (0.75, 1.25, 70, 1.702, False)
    assert a.block.params["eps"] == 1e-4 and plan.head.params["soft_cap"] == 21.0 and plan.tied
    names = {n: s.shape for n, s in expected_tensors(plan).items()}
    assert names["l0.mix.q"] == (4 * 48, 128) and names["l0.mix.dkv"] == (80, 128) and names["l0.mix.g"] == (4, 128) and names["l0.mix.uk"] == (128, 64)
    assert names["l1.mix.dq"] == (56, 128) and names["l1.mix.dq.norm"] == (56,) and names["l1.mix.uq"] == (96, 56) and names["l1.mix.dkv"] == (64, 128)
    assert names["l1.mix.sink"] == (2,) and "l1.mix.q" not in names and "l1.mix.g" not in names and "l0.mix.sink" not in names
    assert names["l0.mlp.e11.down"] == (128, 40) and names["l0.mlp.shared.up"] == (70, 128) and "head" not in names
    assert {"l0.norm1", "l0.norm1b", "l0.norm2", "l0.norm2b", "final.norm", "embed"} <= set(names)
    again, _ = config_from_dict(cfg.to_dict())
    assert again == cfg


def test_what_the_file_leaves_out_does_not_exist():
    bare = [without(LAT, "mixer.rot", "mlp.shared", "mlp.router.groups", "mlp.expert.limit"), without(WIN, "mixer.mask", "mlp"),
            without(LAT, "mixer.rot.scaling", "mlp.shared.limit")]
    d = config(bare)
    d.pop("logit_softcap")
    cfg, plan = config_from_dict(d)
    assert plan.layers[0].mixer.params["position"] is None and plan.layers[1].mixer.params["window"] == 0 and plan.layers[1].feed_forward is None
    ff = plan.layers[0].feed_forward.params
    assert ff["limit"] is None and "shared_ff" not in ff and (ff["groups"], ff["keep_groups"]) == (1, 1)
    assert plan.layers[2].mixer.params["position"].params["scaling"] is None and plan.layers[2].feed_forward.params["shared_limit"] is None
    assert not plan.head.params["soft_cap"]
    names = expected_tensors(plan)
    assert not any("l0.mlp.shared" in n or n.startswith("l1.norm2") for n in names) and {"l1.norm2", "l1.norm2b"} <= set(plan.unread_tensors)
    assert config_from_dict(cfg.to_dict())[0] == cfg


@pytest.mark.parametrize("change,key", [
    (lambda c: c["layers"][0].update(type="attention"), "mixer type"),
    (lambda c: c["layers"][0]["mixer"].pop("kv_rank"), "kv_rank"),
    (lambda c: c["layers"][0]["mixer"].update(dim=0), "positive"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=18), "rot"),
    (lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("fast"), "fast"),
    (lambda c: c["layers"][1]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "mask"),
    (lambda c: c["layers"][0]["mlp"].update(kind="dense"), "feed-forward kind"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=13), "top"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=7), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(count=5), "groups"),
    (lambda c: c["layers"][0]["mlp"]["router"]["groups"].update(keep=5), "groups"),
    (lambda c: c["layers"][0]["mlp"]["expert"].update(ff=0), "positive"),
    (lambda c: c.update(logit_softcap=0.0), "logit_softcap"),
    (lambda c: c.pop("width"), "width"),
])
def test_faults_name_their_key(change, key):
    c = config()
    change(c)
    with pytest.raises(ConfigError, match=key):
        config_from_dict(c)


def test_only_the_compressed_rows_are_kept():
    from cellm_b200.parts.registry import part_class
    _, plan = config_from_dict(config())
    needs = [part_class("mixer", l.mixer.kind).cache_need(l.mixer.params) for l in plan.layers]
    assert needs == [PagedKV(1, 80, 0, values=False), PagedKV(1, 64, 9, values=False)]


def names_of(rec):
    return [n.replace("cellm_", "") for n in rec.names()]


def test_kernels_of_a_decode_step(monkeypatch):
    """Three requests' single tokens: every norm behind a sublayer is one kernel with the sum and the next norm, in the layers, at
    the layers' border and in front of the output; nothing runs in Python."""
    rec = Recorder(monkeypatch)
    cfg, plan, model = zero_model(config())
    run_step(model, plan, [1, 1, 1], [40, 7, 300])
    experts = ["gemm_tcgen05", "route_softmax_all", "experts_gated_rowwise"]
    assert names_of(rec) == [
        "embed", "add_rmsnorm",
        "gemm_tcgen05", "latent_prep", "head_product", "attention_latent", "head_product", "gemm_tcgen05", "norm_add_norm", *experts, "norm_add_norm",
        "gemm_tcgen05", "latent_prep", "gemm_tcgen05", "head_product", "attention_latent", "head_product", "gemm_tcgen05", "norm_add_norm", *experts,
        "norm_add_norm", "gemm_tcgen05", "soft_cap"]
    assert model.program.all_native
    p0, p1 = rec.of("cellm_latent_prep")
    assert p0[0] is None and p0[3] is None and p0[4] is not None and p0[33] == 1 | 4 and p0[10] == 0            # no copy, no query latent, gates, latent and queries
    assert (p0[12], p0[13], p0[6]) == (4 * 48, 4 * 48 + 80, 280) and abs(p0[32] - 1.0693147) < 1e-6            # where the latent and the gates lie; cos and sin
    assert p1[33] == 1 | 2 and (p1[10], p1[12], p1[13]) == (56, 56, -1) and p1[3] is not None and p1[4] is None
    a0, a1 = rec.of("cellm_attention_latent")
    assert a0[19] == 0 and a0[20] is None and a0[21] is not None and a1[19] == 9 and a1[20] is not None and a1[21] is None    # window, sinks, gate
    assert [h[4:6] for h in rec.of("cellm_head_product")[:1]] == [(280, 48)]                                    # queries read where the product left them
    e = rec.of("cellm_experts_gated_rowwise")[0]
    assert e[18] == 1 and [round(v, 4) for v in e[19:22]] == [0.75, 1.25, 1.702]
    assert [r[9:11] for r in rec.of("cellm_route_softmax_all")] == [(3, 4)] * 2 and rec.of("cellm_route_softmax_all")[0][11] == 2
    last = rec.of("cellm_norm_add_norm")[-1]
    assert last[7] is not None and last[8] == 3 and rec.of("cellm_norm_add_norm")[0][7] is None                # the wanted rows only
    cap = rec.of("cellm_soft_cap")[0]
    assert (cap[1], cap[2]) == (3 * 90, 21.0)


def test_kernels_of_a_prompt_step_and_in_thirty_two_bit(monkeypatch):
    rec = Recorder(monkeypatch)
    cfg, plan, model = zero_model(config())
    run_step(model, plan, [300], [0])
    assert names_of(rec).count("head_product_mma") == 4 and "head_product" not in names_of(rec)
    g = rec.of("cellm_gemm_grouped_gated_tcgen05")[0]
    assert g[12] == 1 and round(g[13], 4) == 0.75
    shared = rec.of("cellm_gemm_gated_tcgen05")[0]
    assert shared[12] == 1 and round(shared[13], 4) == 1.25 and round(shared[14], 4) == 1.702
    rec.calls.clear()
    cfg, plan, model = zero_model(config(), dtype=torch.float32)
    run_step(model, plan, [5, 1], [0, 19])
    names = set(names_of(rec))
    assert "attention_plain_masked" in names and not names & {"attention_latent", "gemm_tcgen05", "attention_plain", "moe_sort"}
    m0, m1 = rec.of("cellm_attention_plain_masked")
    assert m0[22] is not None and m0[23] == 4 and m0[17] == 0 and m1[22] is None and m1[19] is not None and m1[17] == 9


def test_a_results_norm_meets_whatever_comes_next(monkeypatch):
    """The next norm in groups, of another element type, or a part in Python: the result is normed and added by a kernel of its own."""
    from cellm_b200.parts.base import FeedForward
    from cellm_b200.parts.routed_experts import RoutedExperts
    rec = Recorder(monkeypatch)
    cfg, plan, model = zero_model(config([LAT]))
    model.final_norm.groups = 2
    run_step(model, plan, [1], [3])
    assert names_of(rec)[-4:] == ["gated_norm_add", "add_rmsnorm", "gemm_tcgen05", "soft_cap"] and names_of(rec).count("norm_add_norm") == 1
    rec.calls.clear()
    cfg, plan, model = zero_model(config([LAT]))
    block = model.blocks[0]
    block.w1 = block.w1.float()
    run_step(model, plan, [1], [3])
    assert names_of(rec).count("gated_norm_add") == 1 and names_of(rec).count("norm_add_norm") == 1
    assert rec.of("cellm_gated_norm_add")[0][8] == 0                       # that norm's weight is 32-bit
    rec.calls.clear()
    monkeypatch.setattr(RoutedExperts, "emit", FeedForward.emit)           # a feed-forward in Python between native norms
    cfg, plan, model = zero_model(config([LAT]))
    run_step(model, plan, [1], [3])
    assert names_of(rec).count("norm_add_norm") == 2 and not model.program.all_native


def test_parts_refuse_what_they_cannot_run():
    from cellm_b200.parts.block import SandwichNormBlock
    from cellm_b200.parts.embedding import LinearHead
    from cellm_b200.parts.norm import RMSNorm
    from cellm_b200.parts.routed_experts import RoutedExperts
    z = lambda *s: torch.zeros(*s)
    w = {"router": z(4, 8), **{f"{k}_{e}": z(*((8, 4) if k == "down" else (4, 8))) for e in range(4) for k in ("gate", "up", "down")}}
    p = {"hidden_size": 8, "experts": 4, "top": 2, "ff_dim": 4, "correction": False}
    with pytest.raises(ConfigError, match="clamped gate belongs"):
        RoutedExperts({**p, "activation": "clamped"}, w, torch.float32)
    with pytest.raises(ConfigError, match="choices"):
        RoutedExperts({**p, "gated": True, "activation": "clamped", "scores": "softmax_all", "groups": 4, "keep_groups": 1}, w, torch.float32)
    ok = RoutedExperts({**p, "gated": True, "activation": "clamped", "scores": "softmax_all", "groups": 4, "keep_groups": 2}, w, torch.float32)
    assert ok.softmax == 2 and ok.limit == float("inf")
    norm = lambda: RMSNorm({"dim": 4, "eps": 1e-5}, {"weight": torch.ones(4)}, torch.bfloat16)
    with pytest.raises(ConfigError, match="together"):
        SandwichNormBlock(norm(), None, norm(), None, {"eps": 1e-5}, {"mixer_result_norm": torch.ones(4)}, torch.bfloat16)
    with pytest.raises(ConfigError, match="soft_cap"):
        LinearHead({"soft_cap": -1.0}, {"weight": z(4, 8)}, torch.float32)


def test_a_long_portion_expands_its_keys_once(monkeypatch):
    """Tokens that fill the tiles: the rows out of their pages, one product for all heads' keys and values, the attention over
    them, and none of the per-head products; the windowed layer takes only the rows that its first new token can see. Short
    portions, single tokens, and portions with far more rows than tokens stay on the rows themselves."""
    rec = Recorder(monkeypatch, hooks={"cellm_attention_expanded_supports": lambda *a: 1})
    cfg, plan, model = zero_model(config())
    run_step(model, plan, [2000, 600, 30], [100, 0, 64])
    names = names_of(rec)
    assert not {"attention_latent", "head_product", "head_product_mma"} & set(names)
    rows = rec.of("cellm_latent_rows")
    assert [r[7] for r in rows] == [2100 + 600 + 94, 2000 + 8 + 600 + 30 + 8] and [r[10] for r in rows] == [0, 9]
    a0, a1 = rec.of("cellm_attention_expanded")
    assert (a0[8], a0[9], a0[10], a0[11]) == (3, 2630, 8 + 3 + 1, 2794) and a0[12:17] == (4, 32, 16, 24, 64) and a0[20] is not None and a0[19] is None
    assert a1[12:17] == (2, 48, 0, 40, 64) and a1[18] == 9 and a1[19] is not None and a1[20] is None
    kv = [g for g in rec.of("cellm_gemm_tcgen05") if (g[3], g[4], g[5]) == (2794, 4 * 56, 64)]
    assert len(kv) == 1 and kv[0][6] == 80                                  # the rows' first 64 columns, 80 apart
    prep = rec.of("cellm_latent_prep")[0]
    assert prep[2] == 16 and prep[1] is not None                            # turned query parts by themselves, head behind head
    for q_lens, ctx_lens in (([100], [0]), ([1] * 8, [500] * 8), ([2300], [40000])):
        rec.calls.clear()
        cfg, plan, model = zero_model(config())
        run_step(model, plan, q_lens, ctx_lens)
        assert len(rec.of("cellm_attention_expanded")) == (1 if ctx_lens == [40000] else 0), (q_lens, ctx_lens)      # the window leaves few rows
