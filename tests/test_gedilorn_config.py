"""Gedilorn on the CPU: the configuration reader, the model description built from it, the manifest of tensors, what
the model keeps between steps, the rotation's frequencies, and the plain model's own consistency."""

import copy
import math

import pytest
import torch

import gedilorn_tiny as gt
import plain_gedilorn as pg


def build(cfg):
    from mini_infer_b200.config import build_model_spec
    from mini_infer_b200.engine.model import Model
    return Model(build_model_spec(cfg))


def owner_of(cfg, i):
    while cfg["layers"][i].get("weights_of") is not None:
        i = cfg["layers"][i]["weights_of"]
    return i


@pytest.mark.parametrize("name", sorted(gt.CONFIGS))
def test_the_description_follows_the_configuration(name):
    cfg = gt.CONFIGS[name]
    model = build(cfg)
    spec = model.spec
    owners = [i for i, l in enumerate(cfg["layers"]) if l.get("weights_of") is None]
    assert [l.name for l in spec.layers] == [f"l{i}" for i in owners]
    assert [owners[e.layer] for e in spec.schedule] == [owner_of(cfg, i) for i in range(len(cfg["layers"]))]
    # every run of a layer owns a cache, whoever owns its weights; the embedding keeps token ids behind a window of two
    latent = [g for g in model.kv_groups if hasattr(g.need, "rank")]
    assert sum(g.num_layers for g in latent) == len(cfg["layers"])
    assert all(g.window == 0 for g in latent)
    slots = {(b["mixer"].group, b["mixer"].layer_slot) for b in model.bindings}
    assert len(slots) == len(cfg["layers"]) and all(b["mixer"].writes for b in model.bindings)
    token = [g for g in model.kv_groups if not hasattr(g.need, "rank")]
    assert len(token) == 1 and token[0].window == 2 and model.embedding_binding.kind == "kv"
    assert not model.state_needs                  # nothing that a dropped step would have to take back
    # the engine's manifest is exactly what the configuration implies
    want = {k: tuple(v.shape) for k, v in gt.make_weights(cfg, 0).items()}
    assert {d.name: tuple(d.shape) for d in model.tensor_decls()} == want


def test_two_token_pages_are_given_back_as_the_request_grows():
    from mini_infer_b200.cache import CacheGroupSpec, CacheManager
    from mini_infer_b200.cache.needs import TokenNeed
    cm = CacheManager([CacheGroupSpec(TokenNeed(window=2), ("a",))], [8], page_size=4, num_slots=1)
    cm.add_request("x")
    total = 0
    for n in (3, 1, 1, 7, 4, 1, 5):
        cm.reserve("x", n)
        cm.commit("x")
        total += n
        cm.check_invariants()
        table = cm.block_table(0, "x")
        # the token before the next one can still be read, and of the pages before its own none is held
        assert table[(total - 1) // 4] >= 0
        assert all(p < 0 for p in table[:(total - 1) // 4])
    cm.release("x")
    assert cm.used_pages() == [0]


@pytest.mark.parametrize("damage", [
    lambda c: c.pop("width"), lambda c: c.pop("streams"), lambda c: c.pop("logit_scale"), lambda c: c.update(streams=0),
    lambda c: c["norm"].pop("eps"), lambda c: c["embedding"].pop("scale"),
    lambda c: c["embedding"]["bigram"].pop("buckets"), lambda c: c["embedding"]["bigram"].update(mul_cur=-1),
    lambda c: c["layers"][0].update(type="attention"), lambda c: c["layers"][0]["mixer"].pop("kv_rank"),
    lambda c: c["layers"][0]["mixer"].update(heads=2.5), lambda c: c["layers"][0]["mixer"].update(scale=0.0),
    lambda c: c["layers"][0]["mixer"].pop("rot"), lambda c: c["layers"][0]["mixer"]["rot"].update(dims=2),
    lambda c: c["layers"][0]["mixer"]["rot"]["scaling"].pop("slow"),
    lambda c: c["layers"][3]["mixer"].update(rot_dim=3),
    lambda c: c["layers"][3]["mlp"].update(kind="moe"), lambda c: c["layers"][3]["mlp"].pop("ff"),
    lambda c: c["layers"][2].update(weights_of=9), lambda c: c["layers"][2].update(weights_of=2),
    lambda c: c["layers"][2].update(weights_of=1),                # another mixer
    lambda c: c["layers"][2].update(mlp=None),                    # another feed-forward than its owner's
    lambda c: c["layers"][2].update(type=gt.PLAIN), lambda c: c.update(layers=[])])
def test_a_damaged_configuration_is_refused(damage):
    from mini_infer_b200.config import ConfigError, build_model_spec
    cfg = copy.deepcopy(gt.CONFIG_A)
    build_model_spec(cfg)
    damage(cfg)
    with pytest.raises(ConfigError):
        build_model_spec(cfg)


def test_shared_weights_that_name_each_other_are_refused():
    from mini_infer_b200.config import ConfigError, build_model_spec
    cfg = copy.deepcopy(gt.CONFIG_B)
    cfg["layers"][2]["weights_of"] = 4
    with pytest.raises(ConfigError):
        build_model_spec(cfg)


def test_a_model_without_a_second_table_keeps_no_token_ids():
    cfg = copy.deepcopy(gt.CONFIG_A)
    cfg["embedding"]["bigram"] = None
    model = build(cfg)
    assert model.embedding_binding is None and all(hasattr(g.need, "rank") for g in model.kv_groups)
    assert "bigram" not in {d.name for d in model.tensor_decls()}


def test_blocks_and_embedding_must_agree_on_the_streams():
    import dataclasses
    from mini_infer_b200.config import build_model_spec
    from mini_infer_b200.config.spec import PartSpec
    from mini_infer_b200.engine.model import Model
    spec = build_model_spec(gt.CONFIG_A)
    emb = PartSpec("token_embedding", dict(spec.embedding.params, streams=3))
    with pytest.raises(ValueError, match="streams"):
        Model(dataclasses.replace(spec, embedding=emb))


def test_a_model_names_the_kernel_sources_it_needs():
    from mini_infer_b200.csrc import build as B
    from mini_infer_b200.ops.library import ENGINE_SOURCES
    files = set(build(gt.CONFIG_B).kernel_files())
    assert {"attention_latent.cu", "attention_shared.cu", "attention_prefill_tc.cu", "residual_streams.cu"} <= files
    assert not files & {"recurrent.cu", "attention.cu", "attention_prefill.cu", "moe.cu", "moe_tc.cu", "residual_forms.cu"}
    assert files | set(ENGINE_SOURCES) <= set(B.sources())


# --------------------------------------------------------------------------- #
# the rotation
# --------------------------------------------------------------------------- #

@pytest.mark.parametrize("dims,base,scaling", [
    (20, 10000.0, (6.0, 1024, 32.0, 1.0)), (64, 100000.0, (40.0, 4096, 32.0, 1.0)), (4, 100.0, (4.0, 64, 8.0, 0.5)),
    (2, 50.0, (2.0, 16, 4.0, 1.0)), (32, 500.0, (3.0, 100, 1.0, 1.0)), (8, 10000.0, (2.0, 16, 1e9, 1e-9)),
    (24, 30.0, (16.0, 1 << 20, 1.0, 0.5)), (12, 1e6, (1.0, 512, 32.0, 1.0))])
def test_yarn_frequencies(dims, base, scaling):
    from mini_infer_b200.config.registry import part_class
    keys = dict(zip(("factor", "original", "fast", "slow"), scaling))
    part = part_class("position", "rope_yarn")(dict(keys, head_dim=dims, theta=base, pairing="neighbours"))
    f, mag = pg.yarn_frequencies(dims, base, keys)
    got = part.table("cpu").double()
    assert torch.allclose(got, torch.tensor(f, dtype=torch.float64), rtol=1e-6)
    assert part.magnitude == pytest.approx(mag) == pytest.approx(0.1 * math.log(scaling[0]) + 1.0)


def test_yarn_leaves_fast_pairs_and_divides_slow_ones():
    f, _ = pg.yarn_frequencies(64, 10000.0, {"factor": 8.0, "original": 4096, "fast": 32.0, "slow": 1.0})
    plain, one = pg.yarn_frequencies(64, 10000.0, None)
    assert one == 1.0 and f[0] == plain[0] and f[-1] == pytest.approx(plain[-1] / 8.0)
    ratio = [a / b for a, b in zip(f, plain)]
    assert all(a >= b for a, b in zip(ratio, ratio[1:])) and any(0.2 < x < 0.9 for x in ratio)


def test_a_mixer_that_cannot_stretch_a_rotation_refuses_it():
    from mini_infer_b200.config.registry import part_class
    from mini_infer_b200.config.spec import PartSpec
    from mini_infer_b200.parts import Runtime, precision_from_name
    pos = PartSpec("rope_yarn", {"head_dim": 8, "theta": 100.0, "factor": 4.0, "original": 64, "fast": 8.0, "slow": 1.0})
    part = part_class("mixer", "gqa_attention")({"hidden_size": 16, "num_heads": 2, "num_kv_heads": 1, "head_dim": 8,
                                                 "position": pos}, "m.")
    t = {d.name: torch.zeros(d.shape) for d in part.tensor_decls()}
    with pytest.raises(ValueError, match="stretch"):
        part.load(t, Runtime(precision_from_name("float32"), torch.device("cpu")))


# --------------------------------------------------------------------------- #
# the plain model
# --------------------------------------------------------------------------- #

@pytest.mark.parametrize("name", sorted(gt.CONFIGS))
def test_plain_model_prefix_property(name):
    """Causal: the logits of a prefix do not change when tokens follow."""
    cfg = gt.CONFIGS[name]
    w = gt.make_weights(cfg, 3)
    toks = gt.random_requests(cfg, [40], 5)["r0"]
    full, part = pg.forward(cfg, w, toks), pg.forward(cfg, w, toks[:23])
    assert torch.allclose(full[:23], part, atol=1e-9)
    assert bool(torch.isfinite(full).all()) and 0.05 < float(full.std()) < 50.0


def test_plain_bigram_rows():
    b = {"buckets": 10, "mul_prev": 3, "mul_cur": 7}
    assert pg.bigram_rows([4, 4, 9], b) == [10, (12 + 28) % 10, (12 + 63) % 10]


def test_plain_streams_update_reads_the_old_streams_and_goes_from_row_to_column():
    xs = torch.tensor([[[1.0], [10.0]]], dtype=torch.float64)
    mix = torch.tensor([[0.0, 2.0], [0.0, 0.0]], dtype=torch.float64)      # from stream 0 to stream 1 only
    got = pg.streams_update(xs, mix, torch.tensor([5.0, 0.0], dtype=torch.float64), torch.tensor([[3.0]], dtype=torch.float64))
    assert got.flatten().tolist() == [15.0, 2.0]


def test_plain_latent_attention_equals_its_folded_form():
    """Folding the key matrices into the queries and applying the value matrices after the weighted sum gives the
    output of the heads' own keys and values."""
    cfg = gt.CONFIG_A
    w = {k: v.double() for k, v in gt.make_weights(cfg, 4).items()}
    m, p, T = cfg["layers"][0]["mixer"], "l0.mix.", 19
    H, d, r, e, c = m["heads"], m["dim"], m["rot_dim"], m["vdim"], m["kv_rank"]
    h = torch.randn(T, cfg["width"], dtype=torch.float64, generator=torch.Generator().manual_seed(1))
    want = pg.latent_attention_mixer(h, w, p, m, 1e-5, True)
    f, mag = pg.yarn_frequencies(r, m["rot"]["base"], m["rot"]["scaling"])
    q = (h @ w[p + "q"].T).view(T, H, d + r)
    dkv = h @ w[p + "dkv"].T
    lat = pg.rms_norm(dkv[:, :c], w[p + "dkv.norm"], 1e-5)
    rows = torch.cat([lat, pg.rotate_neighbours(dkv[:, None, c:], f, mag)[:, 0]], dim=-1)
    folded = torch.einsum("thd,hdc->thc", q[..., :d], w[p + "uk"].view(H, d, c))
    qq = torch.cat([folded, pg.rotate_neighbours(q[..., d:], f, mag)], dim=-1)
    o = pg.causal_softmax_attention(qq, rows[:, None].expand(T, H, c + r), lat[:, None].expand(T, H, c), m["scale"])
    v = torch.einsum("thc,hec->the", o, w[p + "uv"].view(H, e, c)).reshape(T, H * e)
    assert torch.allclose((v * torch.sigmoid(h @ w[p + "g"].T)) @ w[p + "o"].T, want, atol=1e-9)


def test_random_configurations_are_described():
    for seed in range(30):
        cfg = gt.random_config(seed)
        want = {k: tuple(v.shape) for k, v in gt.make_weights(cfg, 0).items()}
        assert {d.name: tuple(d.shape) for d in build(cfg).tensor_decls()} == want
