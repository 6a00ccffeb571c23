"""The Dinatar configuration on the CPU: the keys it reads, what it refuses, the description it builds, what the cache manager
is asked for, and the pages that a window with kept positions gives back."""
import copy

import pytest

from dinatar_helpers import CONFIGS, config, dense, gla, hgrn2, layer, left, lively_tensors, par, right, write_model


def load(cfg, names=None):
    from beglin_b200.config import load_config
    return load_config(copy.deepcopy(cfg), tensor_names=names)


def test_every_size_and_constant_is_read_from_the_configuration():
    arch, cfg = load(CONFIGS["odd"][0])
    assert arch.name == "Dinatar" and cfg.norm_eps == 1e-6 and cfg.embed_scale == 1.7 and cfg.logit_scale == 0.6
    spec = arch.build_spec(cfg)
    assert (spec.vocab, spec.hidden, spec.max_positions, spec.position_name, spec.head_name) == (211, 72, 333, "pos", None)
    assert [s.layer for s in spec.order] == [0, 1, 2, 1, 2, 3, 4]
    assert spec.final_norm.kind == "layernorm" and spec.final_norm.shift and spec.final_norm_bias_name == "final.norm.b"
    g, p, h, q = spec.layers[0], spec.layers[1], spec.layers[2], spec.layers[3]
    assert g.block == "parallel_shared" and q.block == "parallel_mixer"
    m = g.mixer
    assert (m.write, m.n_heads, m.dim, m.vdim, m.decay_rank, m.gated, m.query_silu) == ("key", 3, 10, 7, 5, True, False)
    assert m.decay_power == 0.25 and m.query_scale == pytest.approx(10 ** -0.5)
    f = g.feed_forward
    assert (f.experts, f.top, f.intermediate, f.activation, f.router_activation, f.logit_bias) == (5, 2, 20, "swiglu", "softmax_chosen", True)
    assert f.shared.intermediate == 28 and not f.shared.gated and h.feed_forward.shared is None
    l, r = p.mixer.branches
    assert (l.n_heads, l.n_kv_heads, l.head_dim, l.v_head_dim, l.window, l.keep_first, l.qkv_bias, l.scale) == (6, 2, 9, 13, 17, 3, True, 0.4)
    assert l.position.kind == "none" and l.slopes == tuple(2.0 ** (-8.0 * (i + 1) / 6) for i in range(6))
    assert (r.n_heads, r.vdim, r.state, r.groups, r.conv, r.norm_groups, r.eps) == (3, 8, 11, 1, 3, 2, 1e-6)
    assert p.mixer.scales == (0.5, 0.5) and p.mixer.out_norm_eps == 1e-6 and p.feed_forward.activation == "relu2"
    assert (h.mixer.write, h.mixer.query_silu, h.mixer.query_scale, h.mixer.gated) == ("forget", True, 1.0, False)
    assert p.names["mixer.left.q_proj.bias"] == "l1.mix.left.q.b" and p.names["mixer.right.out_norm.weight"] == "l1.mix.right.out"
    assert g.names["feed_forward.router.logit_bias"] == "l0.mlp.router.b" and g.names["mixer.decay_out.bias"] == "l0.mix.a2.b"
    assert load(cfg.to_json_dict())[1] == cfg


def test_the_short_row_of_the_decays_is_as_long_as_its_tensor(tmp_path):
    import torch
    cfg = config(40, 24, 1e-5, [layer(gla(2, 6, 4, 2.0, 11)), layer(gla(1, 6, 4, 2.0, 3))])
    folder = write_model(str(tmp_path / "m"), cfg, lively_tensors(cfg, 0, torch.float32))
    from beglin_b200.config import load_config
    from beglin_b200.weights import Checkpoint, bind
    ckpt = Checkpoint(folder)
    arch, c = load_config(folder, tensor_names={n: ckpt.shape(n) for n in ckpt.names()})
    assert [l.mixer.rank for l in c.layers] == [11, 3]
    assert bind(arch.build_spec(c), ckpt)["l0.mix.a1"].shape == (11, 24)
    ckpt.close()


def test_absent_keys_have_their_plain_meaning():
    arch, cfg = load(config(40, 16, 0.0, [layer(par(left(2, 1, 4, 4, 0.5, window=3), right(1, 4, 4, 1, 1, 1)))]))
    spec = arch.build_spec(cfg)
    assert cfg.loop is None and spec.embed_scale == 1.0 and spec.logit_scale == 1.0
    assert spec.layers[0].mixer.branches[0].keep_first == 0
    cfg2 = load(config(40, 16, 0.0, [layer(par(left(2, 1, 4, 4, 0.5), right(1, 4, 4, 1, 1, 1)))]))[1]
    assert cfg2.layers[0].mixer.left.window is None


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="conv"), "not known"),
    (lambda c: c["layers"][1]["mixer"]["left"].update(kv_heads=4), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["left"]["mask"].update(keep_first=-1), "keep_first"),
    (lambda c: c["layers"][1]["mixer"].pop("right"), "right"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(groups=2), "multiple"),
    (lambda c: c["layers"][1]["mixer"]["right"].update(norm_groups=7), "equal parts"),
    (lambda c: c["layers"][0]["mixer"].update(tau=0.0), "tau"),
    (lambda c: c["layers"][0]["mlp"]["router"].update(top=9), "top"),
    (lambda c: c["layers"][1]["mlp"].update(kind="glu"), "not known"),
    (lambda c: c.update(loop={"start": 3, "stop": 9, "times": 2}), "loop"),
    (lambda c: c.pop("max_positions"), "max_positions"),
    (lambda c: c["norm"].pop("eps"), "eps"),
])
def test_what_is_refused(change, message):
    from beglin_b200.config import ConfigError
    cfg = copy.deepcopy(CONFIGS["odd"][0])
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        load(cfg)


def test_cache_needs_and_the_kept_pages_that_are_never_given_back():
    from beglin_b200.cache.manager import CacheManager
    from beglin_b200.parts import registry
    from beglin_b200.parts.cache_need import CompositeNeed, FixedStateNeed, PagedKVNeed
    cfg = config(50, 32, 1e-5, [layer(par(left(2, 1, 8, 4, 0.3, window=20, keep=17), right(2, 6, 5, 1, 3, 1)), dense(8)),
                                layer(hgrn2(2, 3, 5)), layer(par(left(2, 1, 8, 4, 0.3, window=20), right(2, 6, 5, 1, 3, 1)))])
    arch, c = load(cfg)
    needs = []
    for l in arch.build_spec(c).layers:
        for _, family, cls, pspec in registry.layer_slots(l):
            if family == "mixer":
                needs.append(cls.cache_need(pspec, None) if getattr(cls, "cache_need_takes_context", False) else cls.cache_need(pspec))
    state = FixedStateNeed((2 * 6 * 5 + 2 * (12 + 10),), "float32")
    assert needs == [CompositeNeed((PagedKVNeed(1, 8, 20, 4, None, 17), state)), FixedStateNeed((30,), "float32"),
                     CompositeNeed((PagedKVNeed(1, 8, 20, 4, None, 0), state))]
    m = CacheManager(needs, page_size=16, num_pages=12, max_requests=2)
    m.add_request("a")
    m.reserve([("a", 100)])
    m.commit([("a", 100)])
    free_before = [g.pool.num_free for g in m.kv_groups]
    m.reserve([("a", 101)])            # the window of the query at 100 begins at 81: pages 0 .. 4 lie in front of it, of which the
    m.commit([("a", 101)])             # first group keeps two (positions 0 .. 16)
    assert [g.pool.num_free - f for g, f in zip(m.kv_groups, free_before)] == [3, 5]
    table = m.block_table(0, ["a"])[0]
    assert (table[:2] >= 0).all() and (table[2:5] == -1).all() and (table[5:7] >= 0).all()
    m.reserve([("a", 150)])
    m.commit([("a", 150)])
    assert (m.block_table(0, ["a"])[0][:2] >= 0).all()
    m.check()
    m.release("a")
    assert all(g.pool.num_free == 12 for g in m.kv_groups)
