"""Dedizen without a GPU: the reader of ``config.json`` and its refusals, the description the engine builds from it, the
manifest against names made from the configuration alone, what each layer keeps between steps and for how long, and the
plain model's own consistency (its mechanisms written a second way)."""

import copy
import math

import pytest
import torch

import dedizen_tiny as dt
import plain_dedizen as pd
from mini_infer_b200.cache.manager import CacheGroupSpec, CacheManager
from mini_infer_b200.cache.needs import KVNeed
from mini_infer_b200.config.dedizen_config import DedizenConfig
from mini_infer_b200.config.model_config import ConfigError
from mini_infer_b200.config.registry import build_model_spec, known_architectures
from mini_infer_b200.engine.model import Model


def test_the_architecture_is_registered():
    assert "Dedizen" in known_architectures()


@pytest.mark.parametrize("name", sorted(dt.CONFIGS))
def test_reader_and_description(name):
    cfg = dt.CONFIGS[name]
    c = DedizenConfig.from_json_dict(cfg)
    assert (c.vocab, c.width, c.eps) == (cfg["vocab"], cfg["width"], cfg["norm"]["eps"])
    spec = build_model_spec(cfg)
    assert spec.lm_head.get("tied_to") == "embed" and spec.final_norm.kind == "rmsnorm"
    for l, ls in zip(cfg["layers"], spec.layers):
        m = l["mixer"]
        assert ls.block.kind == "prenorm_residual" and ls.block.get("feed_forward") == (l["mlp"] is not None)
        assert ("feed_forward" in ls.parts) == ("feed_forward_norm" in ls.parts) == (l["mlp"] is not None)
        if l["mlp"] is not None:
            assert ls.feed_forward.kind == "squared_relu_mlp" and ls.feed_forward.get("intermediate_size") == l["mlp"]["ff"]
        if l["type"] == "mlstm":
            assert ls.mixer.kind == "matrix_lstm" and ls.mixer.get("gate_cap") == m["gate_cap"]
            assert [ls.mixer.get(k) for k in ("num_heads", "head_dim", "value_dim")] == [m["heads"], m["dim"], m["vdim"]]
        elif l["type"] == "rglru":
            assert ls.mixer.kind == "gated_lru"
            assert [ls.mixer.get(k) for k in ("width", "blocks", "conv")] == [m["width"], m["blocks"], m["conv"]]
        else:
            a, r = m["left"], m["right"]
            left, right = ls.mixer, ls.mixer_b
            assert ls.block.get("second_mixer") and ls.block.get("mixer_scale") == ls.block.get("second_mixer_scale") == 0.5
            assert left.kind == "head_mix_attention" and left.get("values") == "keys" and left.get("bias")
            assert left.get("chunk") == a["mask"]["size"] and left.get("scale") == a["scale"] and not left.get("head_mix")
            assert left.get("sink") == "learned" and left.get("output_gate") == "heads"
            assert left.get("qk_norm") == {"eps": c.eps, "after_rotation": True, "gain": False}
            pos, rot = left.get("position"), a.get("rot")
            assert pos.kind == ("none" if not rot else "rope_yarn" if rot.get("scaling") else "rope")
            if rot:
                assert (pos.get("rot_dim"), pos.get("theta"), pos.get("pairing")) == (rot["dims"], rot["base"], "neighbours")
            assert right.kind == "fixed_decay_attention" and right.get("decay") == r["decay"]


@pytest.mark.parametrize("name", sorted(dt.CONFIGS))
def test_manifest_matches_names_made_from_the_configuration(name):
    cfg = dt.CONFIGS[name]
    shapes = {k: tuple(v.shape) for k, v in dt.make_weights(cfg, 1).items()}
    assert {d.name: tuple(d.shape) for d in Model(build_model_spec(cfg)).tensor_decls()} == shapes


def test_what_each_layer_keeps_between_steps():
    up = lambda n: -(-n // 4) * 4
    for cfg in dt.CONFIGS.values():
        model = Model(build_model_spec(cfg))
        states = {owner: need.shape[0] for owner, need in model.state_needs}
        kv = []
        for i, l in enumerate(cfg["layers"]):
            m = l["mixer"]
            if l["type"] == "mlstm":
                H, d, e = m["heads"], m["dim"], m["vdim"]
                assert states[(i, "mixer")] == up(H * d * e) + up(H * d) + up(H)
            elif l["type"] == "rglru":
                assert states[(i, "mixer")] >= m["width"] * m["conv"]
            else:
                r, a = m["right"], m["left"]
                assert states[(i, "mixer_b")] == up(r["heads"] * r["dim"] * r["vdim"])
                kv.append((a["kv_heads"], a["dim"], a["mask"]["size"]))
        assert sorted((g.need.num_kv_heads, g.need.head_dim, g.need.chunk) for g in model.kv_groups) == sorted(kv)


@pytest.mark.parametrize("chunk,page", [(10, 8), (8, 8), (3, 8), (1, 4), (21, 4), (64, 16), (7, 1)])
def test_pages_behind_a_chunk_are_given_back(chunk, page):
    """After every step exactly the pages that the next token's chunk touches are held, however the request was fed; what
    was given back cannot be gone back to."""
    for portions in ([1] * 70, [2, 5, 30, 1, 1, 9, 22], [70]):
        c = CacheManager([CacheGroupSpec(KVNeed(1, 8, chunk=chunk), (0,))], [80], page, 1)
        c.add_request("a")
        n = 0
        for p in portions:
            assert c.reserve("a", p) == n
            c.commit("a")
            n += p
            start = n // chunk * chunk                       # the next token's chunk begins here
            table = c.block_table(0, "a")
            assert [i for i, x in enumerate(table) if x >= 0] == list(range(start // page, -(-n // page)))
            c.check_invariants()
        lost = n // chunk * chunk // page * page
        if lost >= chunk and lost >= page:
            with pytest.raises(ValueError):
                c.truncate("a", max(0, lost - 1))
        c.release("a")
        assert c.used_pages() == [0]


def _bad(change):
    cfg = copy.deepcopy(dt.CONFIG_A)
    change(cfg)
    return cfg


@pytest.mark.parametrize("change", [
    lambda c: c.pop("norm"),
    lambda c: c.update(layers=[]),
    lambda c: c["layers"][0].update(type="attention"),
    lambda c: c["layers"][0]["mixer"]["left"].update(kv_heads=3),
    lambda c: c["layers"][0]["mixer"]["left"].update(vdim=13),
    lambda c: c["layers"][0]["mixer"]["left"]["mask"].update(size=0),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=14),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"].update(dims=3),
    lambda c: c["layers"][0]["mixer"]["left"]["rot"]["scaling"].pop("slow"),
    lambda c: c["layers"][0]["mixer"]["left"].update(scale=0.0),
    lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5]),
    lambda c: c["layers"][0]["mixer"]["right"].update(decay=[0.5, 0.5, 1.5]),
    lambda c: c["layers"][1]["mixer"].update(gate_cap=0),
    lambda c: c["layers"][1]["mixer"].pop("vdim"),
    lambda c: c["layers"][1]["mlp"].update(kind="moe"),
    lambda c: c["layers"][2]["mixer"].update(blocks=4),
])
def test_refusals(change):
    with pytest.raises(ConfigError):
        DedizenConfig.from_json_dict(_bad(change))


# ---- the plain model's own consistency ------------------------------------------------------------------- #

@pytest.mark.parametrize("name", sorted(dt.CONFIGS))
def test_plain_model_is_causal(name):
    cfg = dt.CONFIGS[name]
    w = dt.make_weights(cfg, 3)
    toks = dt.random_requests(cfg, [30], 1)["r0"]
    full = pd.forward(cfg, w, toks)
    assert float((pd.forward(cfg, w, toks[:17]) - full[:17]).abs().max()) < 1e-9


def test_matrix_memory_as_a_sum_over_earlier_tokens():
    """Without the running maximum: ``S_t = sum_j e^(F_t - F_j + i_j) k_j v_j^T``; the maximum m only divides S and n, and
    shows in the normaliser as ``max(|n . q|, 1)`` of the undivided sums."""
    g = torch.Generator().manual_seed(1)
    T, H, d, e = 19, 2, 5, 7
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (d, d, e))
    i = torch.randn(T, H, generator=g, dtype=torch.float64) * 3
    f = pd.log_sigmoid(torch.randn(T, H, generator=g, dtype=torch.float64) * 2)
    got = pd.matrix_memory(q, k, v, i, f)
    F = torch.cumsum(f, dim=0)
    for h in range(H):
        m = 0.0
        for t in range(T):
            m = max(float(f[t, h]) + m, float(i[t, h]))
            a = torch.exp(F[t, h] - F[:t + 1, h] + i[:t + 1, h]) * (k[:t + 1, h] @ q[t, h])
            denom = max(abs(float(a.sum())), 1.0) + 1e-6 * math.exp(m)
            assert torch.allclose(got[t, h], (a @ v[:t + 1, h]) / denom, rtol=1e-9, atol=1e-12)


def test_linear_recurrence_as_a_decayed_sum():
    g = torch.Generator().manual_seed(2)
    T, C = 15, 4
    u, r, i = torch.randn(T, C, generator=g).double(), torch.rand(T, C, generator=g).double(), torch.rand(T, C, generator=g).double()
    lam = torch.randn(C, generator=g).double()
    got = pd.real_gated_lru(u, r, i, lam)
    a = torch.exp(-8 * r * torch.log(1 + torch.exp(lam)))
    for t in range(T):
        want = sum(torch.prod(a[j + 1:t + 1], dim=0) * torch.sqrt(1 - a[j] ** 2) * i[j] * u[j] for j in range(t + 1))
        assert torch.allclose(got[t], want, rtol=1e-9, atol=1e-12)


def test_fixed_decay_as_a_decayed_sum_and_parts_side_by_side():
    g = torch.Generator().manual_seed(3)
    T, H, d, e = 12, 3, 4, 6
    q, k, v = (torch.randn(T, H, n, generator=g, dtype=torch.float64) for n in (d, d, e))
    decay = torch.tensor([0.2, 0.9, 1.0], dtype=torch.float64)
    got = pd.fixed_decay_memory(q, k, v, decay)
    for h in range(H):
        for t in range(T):
            want = sum(decay[h] ** (t - j) * (q[t, h] @ k[j, h]) * v[j, h] for j in range(t + 1))
            assert torch.allclose(got[t, h], want, rtol=1e-9, atol=1e-12)
    w, b, u = torch.randn(2, 3, 3, generator=g).double(), torch.randn(2, 3, generator=g).double(), torch.randn(5, 6, generator=g).double()
    full = torch.block_diag(w[0], w[1])
    assert torch.allclose(pd.block_product(u, w, b), u @ full.T + b.reshape(-1), atol=1e-12)


def test_attention_inside_chunks_token_by_token():
    """Every query alone over the keys of its own chunk, with the rotation as a complex multiplication, a head's values
    the keys before norm and rotation, and the sink in the denominator."""
    g = torch.Generator().manual_seed(4)
    T, W, H, G, d, size = 14, 9, 4, 2, 6, 5
    m = {"heads": H, "kv_heads": G, "dim": d, "vdim": d, "mask": {"size": size}, "scale": 0.8,
         "rot": {"dims": 4, "base": 50.0, "scaling": {"factor": 3.0, "original": 32, "fast": 4.0, "slow": 1.0}}}
    w = {k: torch.randn(*s, generator=g).double() for k, s in
         {"q": (H * d, W), "q.b": (H * d,), "k": (G * d, W), "k.b": (G * d,), "sink": (H,), "g": (H, W), "o": (W, H * d)}.items()}
    h = torch.randn(T, W, generator=g).double()
    got = pd.chunk_attention(h, w, "", m, 1e-5, pd.same)
    freq, mag = pd.yarn(4, m["rot"])

    def turned(x, p):
        z = torch.complex(x[0:4:2], x[1:4:2]) * torch.polar(torch.full((2,), mag, dtype=torch.float64),
                                                            p * torch.tensor(freq, dtype=torch.float64))
        y = torch.cat([torch.stack([z.real, z.imag], dim=1).reshape(4), x[4:]])
        return y / torch.sqrt((y * y).mean() + 1e-5)

    for t in range(T):
        heads = []
        for hd in range(H):
            rows = slice(hd * d, (hd + 1) * d)
            kr = slice(hd // (H // G) * d, (hd // (H // G) + 1) * d)
            q = turned(w["q"][rows] @ h[t] + w["q.b"][rows], t)
            keys = [w["k"][kr] @ h[j] + w["k.b"][kr] for j in range(t // size * size, t + 1)]
            s = torch.stack([m["scale"] * (q @ turned(k, t // size * size + n)) for n, k in enumerate(keys)])
            p = torch.exp(s) / (torch.exp(s).sum() + torch.exp(w["sink"][hd]))
            gate = 1 / (1 + torch.exp(-(w["g"][hd] @ h[t])))
            heads.append(gate * sum(pi * k for pi, k in zip(p, keys)))
        assert torch.allclose(got[t], w["o"] @ torch.cat(heads), rtol=1e-9, atol=1e-10)
