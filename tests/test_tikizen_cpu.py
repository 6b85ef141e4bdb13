"""What the Tikizen design adds that needs no GPU: its configuration reader (what the file leaves out does not exist; faults
name their key), the plan with the items whose cache another item reads and what its pages keep, the tensors the plan
expects, the cache manager's pages for chunks of positions, the layout of joined gate and up rows, what the parts refuse, and
how a block hands the stream on."""
import copy

import numpy as np
import pytest
import torch

from cellm_b200 import models, parts  # noqa: F401  (register architectures and parts)
from cellm_b200.cache import CacheManager
from cellm_b200.cache.native import CacheError
from cellm_b200.config import ConfigError, config_from_dict
from cellm_b200.parts import PagedKV
from cellm_b200.weights.loader import expected_tensors

ROT = {"base": 100.0, "dims": 4, "scaling": {"factor": 2.0, "original": 64, "fast": 8.0, "slow": 1.0}}


def att(**kw):
    return {"type": "attention", "mixer": {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 12, "scale": 0.3, "rot": copy.deepcopy(ROT), **kw}, "mlp": None}


RET = {"type": "retention", "mixer": {"heads": 2, "dim": 6, "vdim": 10, "decay": [0.9, 0.99], "rot": {"base": 50.0, "dims": 4}},
       "mlp": {"kind": "moe", "expert": {"ff": 20}, "router": {"experts": 5, "top": 2}, "shared": {"ff": 30}}}
MAM = {"type": "mamba2", "mixer": {"heads": 4, "vdim": 6, "state": 7, "groups": 2, "norm_groups": 3, "conv": 3}, "mlp": {"kind": "dense", "ff": 24, "limit": 1.25}}


def config(layers, **top):
    return copy.deepcopy({"architecture": "Tikizen", "vocab": 90, "width": 40, "norm": {"eps": 1e-5}, "layers": layers, **top})


def test_the_reader_takes_every_constant_from_the_file():
    d = config([RET, MAM, att(mask={"size": 9}), att(kv_from=2, mask={"size": 9}, heads=8)], postln_alpha=1.75)
    cfg, plan = config_from_dict(d)
    assert cfg.postln_alpha == 1.75 and plan.layers[0].block.params["alpha"] == 1.75
    assert cfg.layers[0].mixer.decay == (0.9, 0.99) and cfg.layers[1].mixer.norm_groups == 3 and cfg.layers[1].mlp.limit == 1.25
    assert cfg.layers[2].mixer.rot.scaling.original == 64 and cfg.layers[2].mixer.chunk == 9
    assert [(e.layer, e.cache_of) for e in plan.order] == [(0, None), (1, None), (2, None), (3, 2)]
    ffn = plan.layers[0].feed_forward.params
    assert (ffn["experts"], ffn["top"], ffn["ff_dim"], ffn["shared_ff"], ffn["scores"], ffn["gated"]) == (5, 2, 20, 30, "softmax", True)
    assert plan.layers[1].feed_forward.params["limit"] == 1.25 and plan.layers[1].feed_forward.params["slope"] == 1.702
    names = expected_tensors(plan)
    assert names["l1.mix.in"].shape == (2 * 24 + 2 * 2 * 7 + 4, 40) and names["l1.mix.conv"].shape == (24 + 28, 3) and names["l1.mix.conv.b"].shape == (52,)
    assert names["l0.mlp.e4.gate"].shape == (20, 40) and names["l0.mlp.shared.sg"].shape == (1, 40) and names["l0.mlp.router.b"].shape == (5,)
    assert names["l3.mix.q"].shape == (64, 40) and "l3.mix.k" not in names and "l3.mix.v" not in names and "l2.mix.k" in names
    assert {"embed", "embed.norm", "final.norm", "head", "l0.norm2"} <= set(names) and "l2.norm2" not in names
    assert "l2.norm2" in plan.unread_tensors
    again, _ = config_from_dict(cfg.to_dict())
    assert again == cfg


def test_what_the_file_leaves_out_does_not_exist():
    bare = {"type": "attention", "mixer": {"heads": 2, "dim": 8, "scale": 0.3}, "mlp": {"kind": "dense", "ff": 8}}
    lone = {"type": "mamba2", "mixer": {"heads": 2, "vdim": 4, "state": 3, "conv": 1}, "mlp": {"kind": "moe", "expert": {"ff": 8}, "router": {"experts": 2, "top": 1}}}
    cfg, plan = config_from_dict(config([bare, lone]))
    m = cfg.layers[0].mixer
    assert (m.kv_heads, m.vdim, m.chunk, m.rot, m.kv_from, cfg.postln_alpha) == (2, 8, 0, None, None, 1.0)
    assert cfg.layers[0].mlp.limit is None and cfg.layers[1].mlp.shared_ff == 0
    assert (cfg.layers[1].mixer.groups, cfg.layers[1].mixer.norm_groups) == (1, 1)
    names = expected_tensors(plan)
    assert not any("shared" in n for n in names) and plan.layers[0].mixer.params["position"] is None


@pytest.mark.parametrize("change,key", [
    (lambda c: c["layers"][0].update(type="conv"), "mixer type"),
    (lambda c: c["layers"][0]["mixer"].update(decay=[0.9]), "decay"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=6), "top"),
    (lambda c: c["layers"][1]["mixer"].update(groups=3), "groups"),
    (lambda c: c["layers"][1]["mixer"].update(norm_groups=5), "norm_groups"),
    (lambda c: c["layers"][1]["mixer"].pop("state"), "state"),
    (lambda c: c["layers"][2]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][2]["mixer"]["rot"].update(dims=10), "rot"),
    (lambda c: c["layers"][2]["mixer"]["rot"]["scaling"].pop("slow"), "slow"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=3), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(kv_from=0), "kv_from"),
    (lambda c: c["layers"][3]["mixer"].update(dim=16), "kv_from"),
    (lambda c: c["layers"][1].update(mlp={"kind": "gated", "ff": 8}), "feed-forward kind"),
    (lambda c: c.pop("width"), "width"),
])
def test_faults_name_their_key(change, key):
    c = config([RET, MAM, att(), att(kv_from=2)])
    change(c)
    with pytest.raises(ConfigError, match=key):
        config_from_dict(c)


@pytest.mark.parametrize("own,readers,kept", [(9, [9], (9, 0)), (9, [], (9, 0)), (9, [20, 4], (0, 20)), (9, [0], (0, 0)), (0, [9], (0, 0)), (30, [9], (0, 30))])
def test_pages_keep_what_the_widest_reader_needs(own, readers, kept):
    mask = lambda n: {"mask": {"size": n}} if n else {}
    cfg, plan = config_from_dict(config([att(**mask(own))] + [att(kv_from=0, **mask(n)) for n in readers]))
    from cellm_b200.parts.registry import part_class
    needs = {part_class("mixer", l.mixer.kind).cache_need(l.mixer.params) for l in plan.layers}
    assert needs == {PagedKV(2, 32, kept[1], chunk=kept[0])}          # rows of 8 and 12 entries widened to one the kernels take
    assert [l.mixer.params["chunk"] for l in plan.layers] == [own] + readers


def test_pages_of_an_ended_chunk_go_back():
    page = 4
    needs = [PagedKV(1, 8, chunk=10), PagedKV(1, 8, window=10), PagedKV(1, 8)]
    cm = CacheManager(needs, [None] * 3, page, 64, 2, torch.float32, "cpu")
    assert len(cm.paged_keys) == 3
    cm.add(1)
    total = 0
    for step in (3, 1, 5, 1, 1, 9, 1, 20, 2, 1, 17):
        assert cm.reserve(1, total + step)
        total += step
        cm.commit(1, total)
        tables = [cm.block_table(1, g, np.full((64,), -1, dtype=np.int32)) for g in range(3)]
        first = total // 10 * 10                                         # the next token's chunk begins here
        for blk in range(-(-total // page)):
            assert (tables[0][blk] >= 0) == ((blk + 1) * page > first), (total, blk)
            assert (tables[1][blk] >= 0) == ((blk + 1) * page > total - 9), (total, blk)
            assert tables[2][blk] >= 0
    assert cm.pages_for(0, 1000, 8) == cm.pages_for(1, 1000, 8) and cm.pages_for(0, 3, 8) == 1
    cm.release(1)
    assert all(cm.free_pages(g) == 64 for g in range(3)) and cm.live == 0
    with pytest.raises(CacheError, match="chunk"):
        CacheManager([PagedKV(1, 8, window=4, chunk=4)], [None], page, 8, 1, torch.float32, "cpu")


def test_gate_and_up_rows_lie_in_blocks():
    from cellm_b200.parts.gated_mlp import blocked_gate_up, widened_columns
    g = torch.arange(70 * 3, dtype=torch.float32).reshape(70, 3) + 1
    both = blocked_gate_up(g, -g)
    assert both.shape == (256, 3)
    assert torch.equal(both[:64], g[:64]) and torch.equal(both[64:128], -g[:64])
    assert torch.equal(both[128:134], g[64:]) and torch.equal(both[192:198], -g[64:]) and not both[134:192].any() and not both[198:].any()
    w = widened_columns(g.T.contiguous())
    assert w.shape == (3, 128) and torch.equal(w[:, :70], g.T) and not w[:, 70:].any()
    assert widened_columns(w).data_ptr() == w.data_ptr()


def test_parts_refuse_what_they_cannot_run():
    from cellm_b200.parts.gated_mlp import GatedMLP
    from cellm_b200.parts.rope import RotaryEmbedding
    from cellm_b200.parts.routed_experts import RoutedExperts
    rope = RotaryEmbedding({"head_dim": 8, "rotary_dim": 8, "theta": 100.0, "scaling": ROT["scaling"]}, "cpu")
    assert rope.amplitude != 1.0 and rope.rotation(amplitude=True)[0] == 8
    with pytest.raises(ConfigError, match="amplitude"):
        rope.rotation()                     # a part that takes no amplitude must not drop it
    z = lambda *s: torch.zeros(*s)
    with pytest.raises(ConfigError, match="biases"):
        GatedMLP({"hidden_size": 8, "ff_dim": 4, "activation": "clamped", "bias": True}, {"gate": z(4, 8), "up": z(4, 8), "down": z(8, 4)}, torch.float32)
    w = {"router": z(2, 8), "correction": z(2), **{f"{k}_{e}": z(*((8, 4) if k == "down" else (4, 8))) for e in range(2) for k in ("gate", "up", "down")}}
    with pytest.raises(ConfigError, match="groups"):
        RoutedExperts({"hidden_size": 8, "experts": 2, "top": 1, "ff_dim": 4, "scores": "softmax", "groups": 2, "keep_groups": 1}, w, torch.float32)
    with pytest.raises(ConfigError, match="scores"):
        RoutedExperts({"hidden_size": 8, "experts": 2, "top": 1, "ff_dim": 4, "scores": "max"}, w, torch.float32)


def test_the_block_hands_the_stream_on_only_to_the_next_item(monkeypatch):
    """The stream in the activations' type is taken from the block of the item before, never from another step or item."""
    from cellm_b200 import ops
    from cellm_b200.parts.base import Residual, StepContext
    from cellm_b200.parts.block import PostNormBlock
    from cellm_b200.parts.norm import RMSNorm
    casts = []
    monkeypatch.setattr(ops, "stream_cast", lambda x, dt: casts.append(1) or x.to(dt))
    monkeypatch.setattr(ops, "post_norm", lambda x, a, alpha, w, eps, dt: x.add_(1).to(dt))

    class Plain:
        def forward(self, h, *rest):
            assert torch.equal(h.float(), stream.x)          # what the sublayer reads is the stream as it is now
            return torch.zeros_like(h)
    norm = lambda: RMSNorm({"dim": 4, "eps": 1e-5}, {"weight": torch.ones(4)}, torch.bfloat16)
    block = PostNormBlock(norm(), Plain(), norm(), Plain(), {"alpha": 2.0}, {}, torch.bfloat16)
    e = torch.zeros(1, dtype=torch.int32)
    ctx = StepContext(T=3, B=1, dtype=torch.bfloat16, device="cpu", token_ids=e, positions=e, seq_of_token=e, cu_seqlens=e, ctx_lens=e, slot_ids=e, err=e)
    stream = Residual(torch.zeros(3, 4))
    for item in (0, 1, 2):
        ctx.extras["order_item"] = item
        block.forward(stream, ctx, None)
    assert len(casts) == 1
    stream.x.zero_()                        # the same context used for another pass
    for item in (0, 1, 3):
        ctx.extras["order_item"] = item
        block.forward(stream, ctx, None)
    assert len(casts) == 3
    with pytest.raises(ConfigError, match="together"):
        PostNormBlock(norm(), Plain(), norm(), None, {}, {}, torch.bfloat16)
