"""The Fanitar configuration on the CPU: the keys it reads, what it refuses, the description it builds, what the cache manager is
asked for; and the plain implementation's own pieces against formulas written another way."""
import copy
import math

import pytest
import torch

from fanitar_helpers import CONFIGS, att, config, dense, lat, layer, lively_tensors, plain, write_model


def load(cfg, names=None):
    from beglin_b200.config import load_config
    return load_config(copy.deepcopy(cfg), tensor_names=names)


def test_every_size_and_constant_is_read_from_the_configuration():
    arch, cfg = load(CONFIGS["odd"][0])
    assert arch.name == "Fanitar" and cfg.norm_eps == 1e-6 and cfg.embed_scale == 1.7 and cfg.logit_scale == 0.6
    spec = arch.build_spec(cfg)
    assert (spec.vocab, spec.hidden, spec.head_name, spec.logit_scale, spec.embed_scale) == (211, 74, "head", 0.6, 1.7)
    assert [(s.layer, s.enter) for s in spec.order] == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None), (4, None)]
    assert [(e.part.index, e.part.again, e.part.passes) for e in spec.entries] == [(0, False, 2), (1, True, 2)]
    a, l, b = spec.layers[0], spec.layers[1], spec.layers[2]
    assert a.block == "sandwich" and b.block == "sandwich_mixer"
    m = a.mixer
    assert (m.n_heads, m.n_kv_heads, m.dim, m.vdim, m.scale, m.diff, m.eps, m.qkv_bias, m.window) == (3, 1, 10, 7, 0.5, 0.3, 1e-6, True, None)
    assert m.position.rotary_dim == 6 and m.position.pairing == "split_half"
    assert m.position.frequencies == tuple(300.0 ** (-2.0 * i / 6) for i in range(3))
    assert b.mixer.position.kind == "none"
    m = l.mixer
    assert (m.n_heads, m.dim, m.rot_dim, m.vdim, m.q_rank, m.kv_rank, m.scale, m.window) == (3, 9, 0, 13, 11, 17, 0.4, 21)
    assert m.gated and m.gate_features and m.sink and spec.layers[3].mixer.window is None
    f = a.feed_forward
    assert (f.intermediate, f.activation, f.limit) == (33, "glu_clamped", 0.7) and l.feed_forward.limit == 2.0
    assert a.names["mixer.k_proj.bias"] == "l0.mix.k.b" and a.names["feed_forward_out_norm.weight"] == "l0.norm2b"
    assert l.names["mixer.gate.weight"] == "l1.mix.g" and l.names["mixer.q_down.norm"] == "l1.mix.dq.norm"
    assert load(cfg.to_json_dict())[1] == cfg


def test_a_query_latent_is_as_long_as_its_tensor_where_the_entry_does_not_say(tmp_path):
    cfg = config(40, 24, 1e-5, [layer(lat(2, 6, 4, 11, 8, 0.5, window=5), dense(8, 1.0)), layer(lat(1, 6, 4, 3, 8, 0.5))])
    tensors = lively_tensors(cfg, 0, torch.float32)
    for l in cfg["layers"]:
        l["mixer"].pop("q_rank")
    folder = write_model(str(tmp_path / "m"), cfg, tensors)
    from beglin_b200.config import ConfigError, load_config
    from beglin_b200.weights import Checkpoint, bind
    ckpt = Checkpoint(folder)
    arch, c = load_config(folder, tensor_names={n: ckpt.shape(n) for n in ckpt.names()})
    assert [l.mixer.q_rank for l in c.layers] == [11, 3]
    assert bind(arch.build_spec(c), ckpt)["l0.mix.dq"].shape == (11, 24)
    ckpt.close()
    with pytest.raises(ConfigError, match="q_rank"):
        load(cfg)


def test_absent_keys_have_their_plain_meaning():
    arch, cfg = load(config(40, 16, 0.0, [layer(att(2, 1, 4, 4, 0.5, 0.1)), layer(lat(1, 4, 4, 4, 4, 0.5))]))
    spec = arch.build_spec(cfg)
    assert cfg.loop is None and spec.embed_scale == 1.0 and spec.logit_scale == 1.0 and not spec.entries
    assert spec.layers[0].mixer.position.kind == "none" and spec.layers[1].mixer.window is None


@pytest.mark.parametrize("change,message", [
    (lambda c: c["layers"][0].update(type="conv"), "not known"),
    (lambda c: c["layers"][0]["mixer"].update(kv_heads=2), "multiple"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=5), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(dims=12), "dims"),
    (lambda c: c["layers"][0]["mixer"]["rot"].update(base=0.0), "base"),
    (lambda c: c["layers"][0]["mixer"].pop("diff"), "diff"),
    (lambda c: c["layers"][0]["mixer"].update(scale=-1.0), "scale"),
    (lambda c: c["layers"][1]["mixer"]["mask"].update(size=0), "size"),
    (lambda c: c["layers"][1]["mixer"].update(kv_rank=0), "kv_rank"),
    (lambda c: c["layers"][0]["mlp"].update(kind="moe"), "not known"),
    (lambda c: c["layers"][0]["mlp"].update(limit=0.0), "limit"),
    (lambda c: c["layers"][0]["mlp"].pop("limit"), "limit"),
    (lambda c: c.update(loop={"start": 3, "stop": 9, "times": 2}), "loop"),
    (lambda c: c.update(loop={"start": 1, "stop": 2, "times": 0}), "loop"),
    (lambda c: c["norm"].pop("eps"), "eps"),
    (lambda c: c.update(layers=[]), "layers"),
])
def test_what_is_refused(change, message):
    from beglin_b200.config import ConfigError
    cfg = copy.deepcopy(CONFIGS["odd"][0])
    change(cfg)
    with pytest.raises(ConfigError, match=message):
        load(cfg)


def test_cache_needs_by_number_format_and_the_pages_a_window_gives_back():
    from beglin_b200.cache.manager import CacheManager
    from beglin_b200.parts import registry
    from beglin_b200.parts.cache_need import PagedKVNeed, PagedLatentNeed
    from beglin_b200.parts.context import BuildContext
    cfg = config(50, 32, 1e-5, [layer(att(2, 1, 24, 40, 0.3, 0.2), dense(8, 1.0)), layer(lat(2, 4, 6, 3, 20, 0.3, window=20)),
                                layer(att(4, 2, 16, 32, 0.3, 0.2)), layer(att(2, 2, 5, 3, 0.3, 0.2)), layer(att(2, 1, 80, 160, 0.1, 0.2))])
    arch, c = load(cfg)

    def needs(dtype):
        ctx, out = BuildContext("cpu", dtype), []
        for l in arch.build_spec(c).layers:
            for _, family, cls, pspec in registry.layer_slots(l):
                if family == "mixer":
                    out.append(cls.cache_need(pspec, ctx) if getattr(cls, "cache_need_takes_context", False) else cls.cache_need(pspec))
        return out
    # a page's key row holds both maps of a kv head
    assert needs(torch.float32) == [PagedKVNeed(1, 48, None, 40), PagedLatentNeed(20, 20), PagedKVNeed(2, 32), PagedKVNeed(2, 10, None, 3),
                                    PagedKVNeed(1, 160)]
    # in bfloat16 as wide as the tensor-core kernels take it, where that does not more than double the cache
    assert needs(torch.bfloat16) == [PagedKVNeed(1, 64), PagedLatentNeed(20, 20), PagedKVNeed(2, 64), PagedKVNeed(2, 10, None, 3),
                                     PagedKVNeed(1, 160)]
    m = CacheManager(needs(torch.float32), page_size=16, num_pages=12, max_requests=2)
    m.add_request("a")
    m.reserve([("a", 100)])
    m.commit([("a", 100)])
    latent = [g for g in m.kv_groups if g.need == PagedLatentNeed(20, 20)][0]
    before = latent.pool.num_free
    m.reserve([("a", 101)])                # the window of the query at 100 begins at 81: pages 0 .. 4 lie in front of it
    m.commit([("a", 101)])
    assert latent.pool.num_free - before == 5
    m.release("a")
    m.check()


# ---------------------------------------------------------------------------------------------- the oracle's own pieces
def test_rotation_depends_on_distance_alone_and_leaves_the_rest():
    g = torch.Generator().manual_seed(1)
    u, v = torch.randn(6, generator=g, dtype=torch.float64), torch.randn(6, generator=g, dtype=torch.float64)
    x = plain.turn_halves(torch.stack([u] * 9), 50.0, 4)
    y = plain.turn_halves(torch.stack([v] * 9), 50.0, 4)
    assert torch.allclose(x[3] @ y[1], x[8] @ y[6]) and not torch.allclose(x[3] @ y[1], x[3] @ y[2])
    assert torch.equal(x[5, 4:], u[4:]) and torch.equal(x[0], u)
    a = 7.0 * 50.0 ** -0.5
    assert torch.allclose(x[7, 1], u[1] * math.cos(a) - u[3] * math.sin(a)) and torch.allclose(x[7, 3], u[3] * math.cos(a) + u[1] * math.sin(a))


def test_a_sink_takes_its_share_once():
    s = torch.tensor([0.3, -1.0, 2.0], dtype=torch.float64)
    b = torch.tensor(0.7, dtype=torch.float64)
    whole = torch.softmax(torch.cat([s, b[None]]), -1)
    assert torch.allclose(plain.plain_softmax_weights(s, b), whole[:3]) and torch.allclose(plain.plain_softmax_weights(s), torch.softmax(s, -1))


def test_the_cut_gate_is_cut_on_the_right_sides():
    z = torch.tensor([-9.0, -0.5, 0.5, 9.0], dtype=torch.float64)
    one = torch.ones(4, dtype=torch.float64)
    sig = lambda t: 1.0 / (1.0 + math.exp(-t))
    got = plain.cut_gate(z, 0.0 * one, 2.0)
    assert torch.allclose(got, torch.tensor([-9.0 * sig(-9.0 * 1.702), -0.5 * sig(-0.851), 0.5 * sig(0.851), 2.0 * sig(3.404)], dtype=torch.float64))
    got = plain.cut_gate(one, z, 2.0)
    assert torch.allclose(got, sig(1.702) * torch.tensor([-1.0, 0.5, 1.5, 3.0], dtype=torch.float64))


def test_the_order_of_runs_and_what_begins_a_pass():
    assert plain.run_order(4, {"start": 1, "stop": 3, "times": 2}) == [(0, None), (1, 0), (2, None), (1, 1), (2, None), (3, None)]
    assert plain.run_order(2, None) == [(0, None), (1, None)]
    assert plain.run_order(2, {"start": 0, "stop": 1, "times": 3}) == [(0, 0), (0, 1), (0, 2), (1, None)]
