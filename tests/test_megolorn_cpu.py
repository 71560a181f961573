"""Host-side checks of the Megolorn design (no GPU): configuration reader and registry, tensor names and shapes, synthetic
weights, and the oracle's mechanisms against closed forms written out in the tests themselves."""
import copy
import json
import math

import pytest
import torch

from moshi_b200.config import DECODER_ARCHITECTURES, DecoderLMConfig, MegolornConfig
from moshi_b200.synth import iter_synth_decoder_tensors
from oracle import megolorn as M

F64 = torch.float64


def small_cfg():
    def mixer(**kw):
        return {"diff": 0.4, "dim": 6, "heads": 4, "kv_heads": 2, "scale": 0.3, "vdim": 5, "mask": {"size": 9},
                "rot": {"base": 100.0, "dims": 4, "scaling": {"factor": 2.0}}, **kw}
    bare = mixer()
    del bare["mask"], bare["rot"]
    return {"architecture": "Megolorn", "embedding": {"scale": 1.5}, "norm": {"eps": 1e-5}, "vocab": 31, "width": 12,
            "layers": [{"type": "attention", "mixer": mixer(), "mlp": {"ff": 9, "kind": "dense", "limit": 0.8}},
                       {"type": "attention", "mixer": mixer(kv_from=0, diff=0.7), "mlp": None},
                       {"type": "attention", "mixer": bare,
                        "mlp": {"expert": {"ff": 7}, "kind": "moe", "router": {"experts": 6, "groups": {"count": 4, "keep": 2}, "identity": 2, "top": 3},
                                "shared": {"ff": 11}}},
                       {"type": "attention", "mixer": mixer(kv_from=0),
                        "mlp": {"expert": {"ff": 8}, "kind": "moe", "router": {"experts": 3, "identity": 0, "top": 1}}}]}


def test_configuration_round_trip_and_registry():
    raw = small_cfg()
    cfg = DecoderLMConfig.from_dict(raw)
    assert isinstance(cfg, MegolornConfig) and DECODER_ARCHITECTURES["Megolorn"] is MegolornConfig
    assert cfg.block == "parallel_residual" and cfg.norm == "layer" and cfg.embedding_scale == 1.5 and not cfg.tied_head
    a, b, c, d = cfg.layers
    assert a.a.kind == "diff_attention" and a.a.chunk == 9 and a.a.qk_norm and a.a.bias and a.a.head_gate and a.a.kv_from == -1
    assert a.a.rot_pairing == "adjacent" and a.a.rot_scaling_kind == "linear" and a.a.rot_scaling == {"factor": 2.0} and a.mlp_kind == "clamped_glu" and a.expert_limit == 0.8
    assert b.a.kv_from == 0 and b.a.diff == 0.7 and b.mlp_kind is None
    assert c.a.chunk == 0 and c.a.rot_dims == 0 and c.experts == 6 and c.identity == 2 and c.groups == 4 and c.groups_keep == 2 and c.shared_ff == 11 and c.top == 3
    assert d.groups == 1 and d.identity == 0 and d.shared_ff == 0
    assert json.loads(json.dumps(cfg.to_dict())) == raw
    from moshi_b200.models.loaders import model_class
    assert model_class(raw).__name__ == "DecoderLM"
    for edit in (lambda x: x["layers"][0].update(type="delta"), lambda x: x["layers"][0]["mlp"].update(kind="other"),
                 lambda x: x["layers"][1]["mixer"].update(kv_from=1), lambda x: x["layers"][3]["mixer"].update(kv_from=1),
                 lambda x: x["layers"][1]["mixer"].update(kv_heads=4)):
        bad = small_cfg()
        edit(bad)
        with pytest.raises(ValueError):
            DecoderLMConfig.from_dict(bad)


def test_tensor_names_and_synthetic_weights():
    cfg = DecoderLMConfig.from_dict(small_cfg())
    s = cfg.tensor_shapes()
    assert s["l0.mix.q"] == (48, 12) and s["l0.mix.k.b"] == (24,) and s["l0.mix.v"] == (10, 12) and s["l0.mix.k.norm"] == (6,) and s["l0.mix.lq2"] == (6,)
    assert s["l0.mix.g"] == (4, 12) and s["l0.mix.o"] == (12, 20) and s["l0.mlp.gate"] == (9, 12) and s["l0.mlp.down"] == (12, 9)
    assert s["l1.mix.q"] == (48, 12) and "l1.mix.k" not in s and "l1.mix.v.b" not in s and "l1.mix.k.norm" not in s and "l1.mlp.up" not in s
    assert s["l2.mlp.router"] == (8, 12) and s["l2.mlp.correction"] == (8,) and s["l2.mlp.e5.up"] == (7, 12) and "l2.mlp.e6.up" not in s
    assert s["l2.mlp.shared.down"] == (12, 11) and "l3.mlp.shared.up" not in s and s["head"] == (31, 12) and s["final.norm"] == (12,)
    t = dict(iter_synth_decoder_tensors(cfg, seed=1))
    assert set(t) == set(s) and all(tuple(t[k].shape) == s[k] for k in s)
    assert float(t["l0.norm1"].float().min()) > 0.5                                        # norm weights sit around one
    lg, layers = M.Oracle(cfg.to_dict(), t).run([3, 1, 4, 1, 5, 9, 2, 6, 5, 3, 5])
    assert lg.shape == (11, 31) and layers.shape == (4, 11, 12) and bool(torch.isfinite(lg).all())


def test_layer_norm_by_hand():
    x = torch.tensor([1.0, 2.0, 6.0], dtype=F64)
    w = torch.tensor([1.0, -2.0, 0.5], dtype=F64)
    var = (4.0 + 1.0 + 9.0) / 3.0
    want = torch.tensor([-2.0, -1.0, 3.0], dtype=F64) / math.sqrt(var + 0.25) * w
    assert torch.allclose(M.layer_norm(x, w, 0.25), want, atol=1e-15)


def test_chunks_are_counted_from_the_start_of_the_sequence():
    assert M.chunk_visible(0, 4) == slice(0, 1) and M.chunk_visible(3, 4) == slice(0, 4) and M.chunk_visible(4, 4) == slice(4, 5)
    assert M.chunk_visible(11, 4) == slice(8, 12) and M.chunk_visible(9, 1) == slice(9, 10) and M.chunk_visible(9, None) == slice(0, 10)


def test_rotation_turns_adjacent_pairs_and_scaling_divides_every_frequency():
    f = M.rotary_frequencies(6, 50.0)
    assert torch.allclose(f, torch.tensor([50.0 ** (-2 * i / 6) for i in range(3)], dtype=F64))
    assert torch.allclose(M.rotary_frequencies(6, 50.0, 4.0), f / 4.0)
    e = torch.zeros(1, 2, 8, dtype=F64)
    e[0, 1, 2] = 1.0
    r = M.rotate_adjacent(e, 3, f)
    assert abs(float(r[0, 1, 2]) - math.cos(3 * float(f[1]))) < 1e-14 and abs(float(r[0, 1, 3]) - math.sin(3 * float(f[1]))) < 1e-14
    g = torch.Generator().manual_seed(0)
    q, k = torch.randn(1, 2, 8, generator=g, dtype=F64), torch.randn(1, 2, 8, generator=g, dtype=F64)
    a = (M.rotate_adjacent(q, 17, f) * M.rotate_adjacent(k, 11, f)).sum()
    b = (M.rotate_adjacent(q, 106, f) * M.rotate_adjacent(k, 100, f)).sum()
    assert abs(float(a - b)) < 1e-10 and torch.equal(M.rotate_adjacent(q, 5, f)[..., 6:], q[..., 6:])


def test_lambda_and_the_combination_of_the_maps():
    p = {"lq1": torch.tensor([0.5, 1.0], dtype=F64), "lk1": torch.tensor([0.2, 0.3], dtype=F64), "lq2": torch.tensor([1.0, 0.0], dtype=F64), "lk2": torch.tensor([-0.5, 9.0], dtype=F64)}
    assert abs(M.diff_lambda(p, 0.3) - (math.exp(0.4) - math.exp(-0.5) + 0.3)) < 1e-14
    a1, a2 = torch.tensor([3.0, 1.0], dtype=F64), torch.tensor([1.0, 1.0], dtype=F64)
    o = torch.tensor([2.0, 0.0], dtype=F64)                                                # lambda = 1
    assert torch.allclose(M.differential_combine(a1, a2, 1.0, 0.25, 0.0), o / math.sqrt(2.0) * 0.75, atol=1e-15)


def test_attention_of_one_head_by_hand():
    """The second token of a chunk: softmax over two keys per map, the difference, the unit norm and the gate, written out."""
    g = torch.Generator().manual_seed(3)
    W, d, dv = 5, 3, 2
    r = lambda *s: torch.randn(*s, generator=g, dtype=F64)
    p = {"q": r(2 * d, W), "q.b": r(2 * d), "k": r(2 * d, W), "k.b": r(2 * d), "v": r(dv, W), "v.b": r(dv), "q.norm": r(d), "k.norm": r(d), "lq1": r(d) * 0.1,
         "lk1": r(d), "lq2": r(d) * 0.1, "lk2": r(d), "g": r(1, W), "o": torch.eye(dv, dtype=F64)}
    m = {"heads": 1, "kv_heads": 1, "dim": d, "vdim": dv, "scale": 0.8, "diff": 0.2, "mask": {"size": 3}}
    hs, st = r(5, W), {}
    for t in range(5):
        out = M.differential_attention(p, m, hs[t], t, st, st, 1e-5)                       # position 4 sees 3 and 4
    unit = lambda u: u / torch.sqrt((u * u).mean() + 1e-5)
    a = []
    for mp in range(2):
        sl = slice(mp * d, (mp + 1) * d)
        q = unit((p["q"] @ hs[4] + p["q.b"])[sl]) * p["q.norm"]
        s = torch.stack([(unit((p["k"] @ hs[j] + p["k.b"])[sl]) * p["k.norm"]) @ q for j in (3, 4)]) * 0.8
        w = torch.softmax(s, 0)
        a.append(w[0] * (p["v"] @ hs[3] + p["v.b"]) + w[1] * (p["v"] @ hs[4] + p["v.b"]))
    lam = math.exp(float(p["lq1"] @ p["lk1"])) - math.exp(float(p["lq2"] @ p["lk2"])) + 0.2
    want = unit(a[0] - lam * a[1]) * 0.8 * torch.sigmoid(p["g"] @ hs[4])
    assert torch.allclose(out, want, atol=1e-12)


def test_router_groups_correction_and_identity():
    z = torch.log(torch.tensor([0.30, 0.05, 0.20, 0.15, 0.10, 0.20], dtype=F64))
    none = torch.zeros(6, dtype=F64)
    idx, w = M.route(z, none, 2, 1, 1)
    assert idx == [0, 2] and abs(w[0] - 0.30) < 1e-12 and abs(w[1] - 0.20) < 1e-12        # not renormalised
    corr = none.clone()
    corr[1] = 1.0
    idx, w = M.route(z, corr, 2, 1, 1)
    assert idx == [1, 0] and abs(w[0] - 0.05) < 1e-12                                       # the correction moves the choice, not the weight
    idx, _ = M.route(z, none, 2, 3, 1)                                                      # groups (0 1) (2 3) (4 5): the first is best, 1 is taken over 2
    assert idx == [0, 1]
    idx, _ = M.route(z - 1.0, none - 5.0, 2, 3, 1)                                          # negative choice scores: the other groups stay out
    assert idx == [0, 1]
    idx, _ = M.route(z, none, 3, 3, 2)
    assert idx == [0, 2, 3]
    # identity experts return the input times their weight; a shared expert is added
    g = torch.Generator().manual_seed(4)
    W, F = 4, 3
    p = {"router": torch.zeros(3, W, dtype=F64), "correction": torch.tensor([0.0, 0.0, 1.0], dtype=F64)}
    for e in ("e0", "e1", "shared"):
        p.update({f"{e}.gate": torch.randn(F, W, generator=g, dtype=F64), f"{e}.up": torch.randn(F, W, generator=g, dtype=F64), f"{e}.down": torch.randn(W, F, generator=g, dtype=F64)})
    h = torch.randn(W, generator=g, dtype=F64)
    mlp = {"router": {"experts": 2, "identity": 1, "top": 1}, "shared": {"ff": F}}
    sh = p["shared.down"] @ (torch.nn.functional.silu(p["shared.gate"] @ h) * (p["shared.up"] @ h))
    assert torch.allclose(M.experts(p, mlp, h), h / 3.0 + sh, atol=1e-12)


def test_bounded_gated_unit_by_hand():
    eye = torch.eye(3, dtype=F64)
    h = torch.tensor([2.0, -3.0, 0.4], dtype=F64)
    y = M.bounded_glu({"gate": eye, "up": -eye, "down": eye}, h, 1.0)
    g, u = [1.0, -3.0, 0.4], [-1.0, 1.0, -0.4]                                              # the gate is bounded above only, the value on both sides
    want = torch.tensor([a / (1 + math.exp(-1.702 * a)) * (b + 1) for a, b in zip(g, u)], dtype=F64)
    assert torch.allclose(y, want, atol=1e-14)


def test_state_is_carried_over_a_cut_and_shared_between_layers():
    cfg = DecoderLMConfig.from_dict(small_cfg())
    t = dict(iter_synth_decoder_tensors(cfg, seed=2))
    o = M.Oracle(cfg.to_dict(), t)
    toks = [3, 7, 7, 1, 0, 30, 12, 5, 9, 2, 2, 8]
    whole, _ = o.run(toks)
    st = o.new_state()
    a, _ = o.run(toks[:4], st)
    b, _ = o.run(toks[4:], st)
    assert torch.equal(torch.cat([a, b]), whole)
    assert "k" in st["layers"][0] and not st["layers"][1] and "k" in st["layers"][2] and not st["layers"][3]
    # a first token of a chunk sees itself alone: what came before does not reach it through chunked layers
    only = copy.deepcopy(cfg.to_dict())
    only["layers"] = only["layers"][:2]
    o2 = M.Oracle(only, {k: v for k, v in t.items() if not k.startswith(("l2", "l3"))})
    x, _ = o2.run(toks)
    y, _ = o2.run([1] * 9 + toks[9:])
    assert torch.equal(x[9:], y[9:]) and not torch.equal(x[8], y[8])
