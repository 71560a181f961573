"""The Megolorn decoder LM on the GPU against its float64 oracle (``oracle/megolorn.py``): every mechanism alone, whole prompts
with every layer's output, prompts in portions down to two tokens, token-by-token decoding, unequal batches, slots given back
and used again, sharp attention at the chunks' edges in prompts and in decoding, far keys, layers that read another layer's keys
and values, the router's groups, correction and identity experts, the first tokens of a sequence, odd and aligned sizes, and
greedy generation through the scheduler and the command line."""
import copy
import json
import subprocess
import sys
from pathlib import Path

import pytest
import torch

from moshi_b200.config import DecoderLMConfig
from moshi_b200.synth import iter_synth_decoder_tensors
from oracle.decoder_lm import logit_error
from oracle.megolorn import F64, Oracle

from .test_gpu_zz_decoder_lm import gen_for, tokens, write_model

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
TOL = {torch.float32: 3e-5, torch.bfloat16: 8e-2}
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])


def attention(heads, kv, dim, vdim, scale, chunk=0, diff=0.5, rot_dims=0, base=300.0, factor=None, kv_from=None, mlp=None):
    m = {"diff": diff, "dim": dim, "heads": heads, "kv_heads": kv, "scale": scale, "vdim": vdim}
    if chunk:
        m["mask"] = {"size": chunk}
    if rot_dims:
        m["rot"] = {"base": base, "dims": rot_dims}
        if factor:
            m["rot"]["scaling"] = {"factor": factor}
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "attention", "mixer": m, "mlp": mlp}


def dense(ff, limit=1.2):
    return {"ff": ff, "kind": "dense", "limit": limit}


def moe(experts, top, ff, identity=0, groups=None, shared=None):
    r = {"experts": experts, "identity": identity, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    d = {"expert": {"ff": ff}, "kind": "moe", "router": r}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def make_cfg(layers, vocab, width, emb=1.5, eps=1e-5):
    return DecoderLMConfig.from_dict({"architecture": "Megolorn", "embedding": {"scale": emb}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width})


# odd sizes: nothing is a multiple of 8; three query heads per key head and one; value size unlike key size; rotation of a part of the
# head, the whole head, none; chunks shorter than the prompts, of one token, and none; layers that read the keys and values of a
# layer further back under a chunk of their own; experts with and without groups, identity and shared experts; a layer without feed-forward
ODD = make_cfg([attention(6, 2, 10, 12, 0.3, chunk=17, diff=0.35, rot_dims=6, factor=3.0, mlp=moe(5, 2, 24, identity=1, groups=(3, 2), shared=19)),
                attention(6, 2, 10, 12, 0.4, chunk=29, diff=0.6, rot_dims=6, factor=3.0, kv_from=0, mlp=dense(30)),
                attention(3, 3, 14, 5, 0.25, diff=0.2, rot_dims=14, base=1e4, mlp=None),
                attention(5, 1, 7, 9, 0.35, chunk=40, diff=0.8, mlp=moe(7, 3, 17, identity=2)),
                attention(3, 3, 14, 5, 0.3, diff=0.45, chunk=11, rot_dims=14, base=1e4, kv_from=2, mlp=moe(3, 1, 21, shared=8)),
                attention(2, 2, 9, 6, 0.3, chunk=23, mlp=dense(13, limit=0.4))], vocab=97, width=52)
# aligned sizes: in bfloat16 every linear takes the tcgen05 GEMM, attention and experts their tensor-core kernels; the order starts with
# experts; one key head for all query heads; more experts per group than kept groups; value columns that fill no accumulator tile
ALIGNED = make_cfg([attention(4, 1, 32, 16, 0.18, chunk=48, diff=0.3, rot_dims=16, factor=8.0, mlp=moe(6, 3, 48, identity=2, groups=(2, 1), shared=64)),
                    attention(8, 2, 16, 48, 0.25, chunk=64, diff=0.55, rot_dims=16, base=1e5, mlp=dense(128)),
                    attention(8, 2, 16, 48, 0.25, chunk=64, diff=0.7, rot_dims=16, base=1e5, kv_from=1, mlp=moe(8, 2, 32, groups=(4, 2), shared=32)),
                    attention(4, 4, 64, 80, 0.12, diff=0.4, rot_dims=32, mlp=dense(96, limit=3.0)),
                    attention(4, 1, 32, 16, 0.18, chunk=33, diff=0.5, rot_dims=16, factor=8.0, kv_from=0, mlp=None)], vocab=200, width=96)


def build(cfg, dtype, seed=3, edit=None):
    from moshi_b200.models import DecoderLM
    tensors = dict(iter_synth_decoder_tensors(cfg, seed=seed))
    if dtype == torch.bfloat16:
        # a bf16 rounding can turn a router's close call and swap an expert for that token; with random weights that happens
        # every few dozen tokens.  Small expert outputs keep such a swap inside the bf16 tolerance (float32 runs as drawn).
        for k in tensors:
            if ".mlp.e" in k and k.endswith(".down"):
                tensors[k] = tensors[k] * 0.25
    if edit:
        edit(tensors)
    return DecoderLM(cfg, tensors, device="cuda:0", dtype=dtype), Oracle(cfg.to_dict(), tensors)


def assert_close(got, want, dtype, what="", tol=None):
    """float32: every row within the tolerance.  bfloat16: a rounding can turn a router's close call, which changes that token
    as a whole, so up to a tenth of the rows may be off while the median stays well inside."""
    e = logit_error(got.cpu(), want)
    tol = tol or TOL[dtype]
    if dtype == torch.float32:
        assert float(e.max()) < tol, f"{what}: relative logit error {float(e.max()):.3g} at row {int(e.argmax())}"
    else:
        assert int((e > tol).sum()) <= max(1, e.numel() // 10) and float(e.median()) < tol, f"{what}: relative logit errors {e.tolist()}"


def in_portions(gen, slot, toks, cuts):
    """The tokens in portions of the given sizes (the rest in one), every row wanted."""
    out, at = [], 0
    for n in list(cuts) + [len(toks)]:
        part = toks[at:at + n]
        if not part:
            break
        out.append(gen.step([(slot, part)], list(range(len(part)))))
        at += len(part)
    return torch.cat(out)


def sharpen(by, names=("q.norm", "k.norm")):
    """Queries and keys are normed, so their norms' weights set how sharp the scores are."""
    def edit(t):
        for k in t:
            if k.endswith(names):
                t[k] = t[k] * by
    return edit


@BOTH
@pytest.mark.parametrize("cfg", [ODD, ALIGNED], ids=["odd", "aligned"])
def test_whole_prompt_and_every_layer(cfg, dtype):
    model, orc = build(cfg, dtype)
    toks = tokens(90, cfg.vocab, 1)
    want, layers = orc.forward(toks, return_layers=True)
    with gen_for(model, trace_layers=True) as gen:
        got = gen.step([(1, toks)], list(range(len(toks))))
        lo = gen.layer_outputs().cpu()
        assert gen.error_flags() == 0
    scale = float(layers.abs().max())
    for i in range(len(cfg.layers)):
        err = ((lo[i].to(F64) - layers[i]).abs().amax(-1) / scale)
        if dtype == torch.float32:
            assert float(err.max()) < 2e-5, f"layer {i}: {float(err.max()):.3g}"
        else:
            assert int((err > 8e-2).sum()) <= 9 and float(err.median()) < 3e-2, f"layer {i}: {err.tolist()}"
    assert_close(got, want, dtype)


ALONE = {
    "attention": [attention(6, 2, 10, 12, 0.3, chunk=13, rot_dims=6)],
    "attention_linear_scaling": [attention(4, 2, 12, 9, 0.3, chunk=30, rot_dims=12, base=50.0, factor=2.5)],
    "attention_factor_one": [attention(2, 2, 8, 8, 0.4, chunk=30, rot_dims=8, factor=1.0)],
    "attention_unrotated": [attention(3, 3, 9, 9, 0.35, chunk=21)],
    "attention_without_a_mask": [attention(4, 1, 8, 6, 0.3, rot_dims=4)],
    "attention_one_head": [attention(1, 1, 16, 4, 0.3, chunk=5, diff=0.1)],
    "attention_dim_one_pair": [attention(2, 1, 2, 3, 0.7, chunk=50, rot_dims=2)],
    "attention_diff_zero": [attention(2, 1, 6, 6, 0.4, chunk=12, diff=0.0)],
    "attention_many_heads_per_key_head": [attention(20, 1, 6, 5, 0.4, chunk=14, rot_dims=6)],
    "attention_of_another_layer": [attention(4, 2, 8, 6, 0.4, chunk=16, rot_dims=8), attention(4, 2, 8, 6, 0.3, chunk=7, diff=0.7, rot_dims=8, kv_from=0),
                                   attention(4, 2, 8, 6, 0.3, diff=0.3, rot_dims=8, kv_from=0)],
    "dense": [attention(1, 1, 2, 2, 0.5, chunk=1, mlp=dense(45, limit=0.6))],
    "dense_wide_limit": [attention(1, 1, 2, 2, 0.5, chunk=1, mlp=dense(40, limit=50.0))],
    "experts": [attention(1, 1, 2, 2, 0.5, chunk=1, mlp=moe(6, 2, 33))],
    "experts_all_chosen": [attention(1, 1, 2, 2, 0.5, chunk=1, mlp=moe(3, 5, 20, identity=2))],
    "experts_top_one_of_one_group": [attention(1, 1, 2, 2, 0.5, chunk=1, mlp=moe(7, 1, 20, identity=1, groups=(4, 1), shared=31))],
    "experts_a_group_of_identities": [attention(1, 1, 2, 2, 0.5, chunk=1, mlp=moe(4, 3, 20, identity=4, groups=(2, 1)))],
    "experts_all_groups_kept": [attention(1, 1, 2, 2, 0.5, chunk=1, mlp=moe(8, 4, 16, groups=(4, 4), shared=16))],
    "experts_fifty": [attention(1, 1, 2, 2, 0.5, chunk=1, mlp=moe(50, 6, 9, identity=10, groups=(6, 3), shared=5))],
}


@pytest.mark.parametrize("what", sorted(ALONE))
def test_mechanisms_in_isolation(what):
    cfg = make_cfg(copy.deepcopy(ALONE[what]), vocab=61, width=44, emb=0.7)
    model, orc = build(cfg, torch.float32, seed=11)
    toks = tokens(70, cfg.vocab, 2)
    with gen_for(model) as gen:
        assert_close(gen.step([(0, toks)], list(range(len(toks)))), orc.forward(toks), torch.float32, what)
        assert_close(in_portions(gen, 1, toks, [41, 2] + [1] * 20), orc.forward(toks), torch.float32, what + ", portions")


@BOTH
@pytest.mark.parametrize("chunk", [1, 2, 7, 32, 33, 64, 65, 97, 128])
def test_sharp_attention_at_the_chunks_edges(chunk, dtype):
    """Large query and key weights make single keys dominate, so a chunk that is one token off shows; the oracle itself moves by
    far more than the tolerance when its chunk changes by one.  bfloat16 takes the tensor-core kernels."""
    # bfloat16 rounds keys and queries: scores as sharp as float32 can take would turn that rounding into the result's error
    cfg = make_cfg([attention(4, 2, 16, 16, 0.5, chunk=chunk, rot_dims=8)], vocab=53, width=48)
    model, orc = build(cfg, dtype, seed=5, edit=sharpen(2.0 if dtype == torch.float32 else 1.2))
    n = max(100, 2 * chunk + 36)                      # edges are passed by prompt tokens and by single tokens
    toks = tokens(n, cfg.vocab, 3)
    want = orc.forward(toks)
    for off in (-1, 1):
        if chunk + off < 1:
            continue
        d = cfg.to_dict()
        d["layers"][0]["mixer"]["mask"]["size"] = chunk + off
        assert float(logit_error(Oracle(d, orc.t).forward(toks), want).max()) > (50 if dtype == torch.float32 else 1.5) * TOL[dtype]
    with gen_for(model, capacity=n + 8, max_step_tokens=max(256, n)) as gen:
        def close(got, what):
            e = logit_error(got.cpu(), want)
            assert float(e.max()) < TOL[dtype], f"{what}: {float(e.max()):.3g} at {int(e.argmax())}"
        close(gen.step([(0, toks)], list(range(n))), "whole")
        gen.release(0)
        close(in_portions(gen, 0, toks, [chunk + 1, 2, 3] + [1] * (chunk + 8 if chunk > 40 else 40) + [2] * 5), "portions and single tokens")
        for split in (2, 5):                          # an edge inside a split of the keys, and splits that a row sees nothing of
            gen.release(0)
            gen.set_option("attn_split", split)
            close(in_portions(gen, 0, toks, [n - 12] + [1] * 12), f"keys cut {split} times")
        gen.set_option("attn_split", 0)


@BOTH
def test_a_far_key_without_a_mask_and_inside_a_long_chunk(dtype):
    """Sharp scores over 600 tokens, so that single keys hundreds of positions back carry rows of the result: in a prompt, in portions,
    and in single tokens, without a mask, and through a layer that reads the same keys inside chunks of 590."""
    cfg = make_cfg([attention(4, 2, 16, 16, 0.5, rot_dims=8), attention(4, 2, 16, 16, 0.6, chunk=590, rot_dims=8, kv_from=0)], vocab=53, width=48)
    model, orc = build(cfg, dtype, seed=6, edit=sharpen(2.0 if dtype == torch.float32 else 1.2))
    toks = tokens(600, cfg.vocab, 5)
    want = orc.forward(toks)
    short = orc.forward(toks[300:])                   # the same last tokens without the first 300: the far keys matter
    assert float(logit_error(short[-40:], want[-40:]).max()) > 50 * TOL[torch.float32]
    with gen_for(model, capacity=640, max_step_tokens=640) as gen:
        assert_close(gen.step([(0, toks)], list(range(600))), want, dtype, "whole")
        gen.release(0)
        assert_close(in_portions(gen, 0, toks, [517, 2, 33] + [1] * 40), want, dtype, "portions and single tokens")


@pytest.mark.parametrize("heads,kv,dim,vdim", [(4, 2, 16, 16), (8, 8, 32, 64), (6, 2, 48, 112), (20, 1, 16, 32), (70, 1, 16, 16), (3, 1, 128, 128), (2, 1, 64, 144), (4, 2, 24, 40)])
def test_both_attention_kernels_in_bfloat16(heads, kv, dim, vdim):
    """Tensor cores and CUDA cores on the same bf16 cache: prompts, single tokens, keys cut over CTAs, tiles that cut a token's heads
    (20 and 70 query heads per key head), and sizes that only the CUDA cores take."""
    cfg = make_cfg([attention(heads, kv, dim, vdim, dim ** -0.5, chunk=90, rot_dims=dim // 4 * 2)], vocab=53, width=64)
    model, orc = build(cfg, torch.bfloat16, seed=7, edit=sharpen(1.5))
    toks = tokens(150, cfg.vocab, 9)
    want = orc.forward(toks)
    got = {}
    with gen_for(model) as gen:
        for tc in (1, 0):
            gen.set_option("attn_tc", tc)
            for split in (0, 1, 3):
                gen.set_option("attn_split", split)
                gen.release(0)
                got[tc, split] = in_portions(gen, 0, toks, [101, 17] + [1] * 25).cpu()
                e = logit_error(got[tc, split], want)
                assert float(e.max()) < TOL[torch.bfloat16], f"attn_tc {tc}, attn_split {split}: {float(e.max()):.3g} at {int(e.argmax())}"
        assert gen.error_flags() == 0


def test_layers_read_the_keys_and_values_of_the_layer_they_name():
    """The oracle moves by far more than the tolerance when a layer reads another source, so agreement means the right cache."""
    def layers(src):
        return [attention(4, 2, 8, 6, 0.5, chunk=20, rot_dims=8), attention(4, 2, 8, 6, 0.5, chunk=20, rot_dims=8),
                attention(4, 2, 8, 6, 0.5, chunk=20, rot_dims=8, kv_from=src), attention(4, 2, 8, 6, 0.5, chunk=31, rot_dims=8, kv_from=1 - src)]
    toks = tokens(80, 53, 14)
    wants = []
    for src in (0, 1):
        cfg = make_cfg(layers(src), vocab=53, width=40)
        model, orc = build(cfg, torch.float32, seed=15)
        wants.append(orc.forward(toks))
        with gen_for(model) as gen:
            assert_close(in_portions(gen, 2, toks, [50, 3] + [1] * 10), wants[-1], torch.float32, f"kv_from {src}")
    assert float(logit_error(wants[1], wants[0]).max()) > 50 * TOL[torch.float32]


def test_router_with_negative_choice_scores_and_a_correction_that_moves_the_choice():
    """All choice scores negative (the groups that are left out must not win with a zero), corrections as large as the scores; the
    oracle moves when the correction or the groups are left out."""
    cfg = make_cfg([attention(2, 1, 6, 6, 0.4, chunk=8, mlp=moe(9, 3, 25, identity=3, groups=(4, 2), shared=10))] * 2, vocab=61, width=44)

    def edit(t):
        for k in t:
            if k.endswith("correction"):
                t[k] = (torch.linspace(-0.9, -0.5, t[k].numel()) - 0.3 * (torch.arange(t[k].numel()) % 3 == 1)).to(t[k].dtype)
            if k.endswith("router"):
                t[k] = t[k] * 3.0
    model, orc = build(cfg, torch.float32, seed=17, edit=edit)
    toks = tokens(120, cfg.vocab, 16)
    want = orc.forward(toks)
    flat = dict(orc.t)
    for k in flat:
        if k.endswith("correction"):
            flat[k] = torch.zeros_like(flat[k])
    assert float(logit_error(Oracle(cfg.to_dict(), flat).forward(toks), want).max()) > 50 * TOL[torch.float32]
    d = cfg.to_dict()
    for L in d["layers"]:
        L["mlp"]["router"].pop("groups")
    assert float(logit_error(Oracle(d, orc.t).forward(toks), want).max()) > 50 * TOL[torch.float32]
    with gen_for(model) as gen:
        assert_close(gen.step([(0, toks)], list(range(120))), want, torch.float32, "whole")
        assert_close(in_portions(gen, 1, toks, [60, 2] + [1] * 20), want, torch.float32, "portions")


@BOTH
@pytest.mark.parametrize("cfg", [ODD, ALIGNED], ids=["odd", "aligned"])
@pytest.mark.parametrize("cuts", [[2, 3, 1, 7, 2, 40], [1] * 12, [5, 4, 3, 2] * 6, [2] * 45, [64]], ids=["ragged", "ones", "cycle", "twos", "long"])
def test_portions_equal_the_whole_prompt(cfg, cuts, dtype):
    model, orc = build(cfg, dtype)
    toks = tokens(130, cfg.vocab, 6)
    want = orc.forward(toks)
    with gen_for(model) as gen:
        assert_close(in_portions(gen, 1, toks, cuts), want, dtype)
        assert gen.error_flags() == 0


@pytest.mark.parametrize("n", [1, 2, 3, 6])
def test_first_tokens_at_once_and_one_by_one(n):
    model, orc = build(ODD, torch.float32)
    toks = tokens(n, ODD.vocab, 20 + n)
    want = orc.forward(toks)
    with gen_for(model) as gen:
        assert_close(gen.step([(0, toks)], list(range(n))), want, torch.float32, "at once")
        assert_close(in_portions(gen, 1, toks, [1] * n), want, torch.float32, "one by one")


@BOTH
def test_long_decoding_token_by_token(dtype):
    cfg = ALIGNED if dtype == torch.bfloat16 else ODD
    model, orc = build(cfg, dtype)
    toks = tokens(190, cfg.vocab, 7)
    want = orc.forward(toks)
    with gen_for(model) as gen:
        assert_close(in_portions(gen, 0, toks, [10] + [1] * 180), want, dtype)
        assert gen.error_flags() == 0


@BOTH
@pytest.mark.parametrize("cfg", [ODD, ALIGNED], ids=["odd", "aligned"])
def test_unequal_batch_equals_each_request_alone(cfg, dtype):
    model, orc = build(cfg, dtype)
    a, b, c = tokens(61, cfg.vocab, 8), tokens(9, cfg.vocab, 9), tokens(35, cfg.vocab, 10)
    wa, wb, wc = orc.forward(a), orc.forward(b + [b[0]]), orc.forward(c)
    with gen_for(model) as gen:
        gen.step([(0, a[:40]), (2, c[:33])], [])
        got = gen.step([(0, a[40:]), (1, b), (2, c[33:34])], list(range(21 + 9 + 1)))      # 21 + 9 + 1 tokens on histories of 40 / 0 / 33
        assert_close(got[:21], wa[40:], dtype, "a")
        assert_close(got[21:30], wb[:9], dtype, "b")
        assert_close(got[30:], wc[33:34], dtype, "c")
        got = gen.step([(1, [b[0]]), (2, [c[34]])], [0, 1])                                  # single tokens of two requests on their histories
        assert_close(got[:1], wb[9:], dtype, "b, one token")
        assert_close(got[1:], wc[34:], dtype, "c, one token")


def test_slots_are_given_back_and_used_again():
    model, orc = build(ODD, torch.float32)
    a, b = tokens(120, ODD.vocab, 12), tokens(11, ODD.vocab, 13)
    with gen_for(model, slots=1) as gen:
        gen.step([(0, a)], [])
        with pytest.raises(RuntimeError):
            gen.step([(0, tokens(200, ODD.vocab, 14))], [])                                 # would overflow the slot: refused whole
        gen.release(0)
        assert gen.slot_length(0) == 0
        assert_close(gen.step([(0, b)], list(range(11))), orc.forward(b), torch.float32)
        gen.release(0)
        assert_close(in_portions(gen, 0, a, [3, 50]), orc.forward(a), torch.float32, "again")


def test_configurations_that_the_handle_refuses():
    from moshi_b200.models import DecoderLM
    for L in (attention(3, 2, 8, 8, 0.3), attention(2, 1, 8, 8, 0.3, rot_dims=10), attention(2, 1, 8, 8, 0.3, mlp=moe(5, 2, 8, groups=(2, 1))),
              attention(2, 1, 8, 8, 0.3, mlp=moe(6, 3, 8, groups=(3, 1))), attention(2, 1, 8, 8, 0.3, mlp=dense(8, limit=0.0))):
        cfg = make_cfg([L], vocab=20, width=16)
        with pytest.raises(ValueError):
            DecoderLM(cfg, {}, device="cuda:0", dtype=torch.float32)


def test_greedy_generation_through_the_scheduler():
    from moshi_b200.serving import TokenScheduler
    cfg = ODD
    model, orc = build(cfg, torch.float32)
    prompts = {"a": tokens(23, cfg.vocab, 40), "b": tokens(3, cfg.vocab, 41), "c": tokens(40, cfg.vocab, 42)}
    with gen_for(model, slots=2, capacity=80, max_step_tokens=32) as gen:      # 3 requests over 2 slots, prompts cut at 32 tokens
        sched = TokenScheduler(gen)
        for k, p in prompts.items():
            sched.submit(k, p, 12)
        out = sched.run()
    for k, p in prompts.items():
        want, gaps = orc.greedy(p, 12)
        for i, (g, w, gap) in enumerate(zip(out[k], want, gaps)):
            if g != w:
                assert gap < 1e-3, f"request {k}: token {i} is {g}, the oracle says {w} with a gap of {gap}"
                break


@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_command_line_replays_steps_and_generates(tmp_path, dtype):
    cfg = ODD if dtype == "float32" else ALIGNED
    tensors = dict(iter_synth_decoder_tensors(cfg, seed=8))
    write_model(tmp_path / "m", cfg, tensors)
    orc = Oracle(cfg.to_dict(), tensors)
    a, b = tokens(30, cfg.vocab, 50), tokens(6, cfg.vocab, 51)
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:21], "want": [0, 20]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[21:], "want": []}], "end": ["a"]},
             {"step": 2, "entries": [{"id": "b", "tokens": b, "want": [5]}], "end": ["b"]}]
    (tmp_path / "out").mkdir()
    r = subprocess.run([str(ROOT / "bin" / "trace_run"), "--model", str(tmp_path / "m"), "--dtype", dtype, "--out", str(tmp_path / "out"),
                        "--max-tokens", "64"], input="\n".join(json.dumps(s) for s in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [l for l in r.stdout.splitlines() if l.startswith("done")] == ["done 0", "done 1", "done 2"]
    import numpy as np
    td = torch.float32 if dtype == "float32" else torch.bfloat16
    got0 = torch.from_numpy(np.fromfile(tmp_path / "out" / "0.f32", dtype="<f4").reshape(2, cfg.vocab))
    got2 = torch.from_numpy(np.fromfile(tmp_path / "out" / "2.f32", dtype="<f4").reshape(1, cfg.vocab))
    assert_close(got0, orc.forward(a)[[0, 20]], td)
    assert_close(got2, orc.forward(b)[[5]], td)
    if dtype == "float32":
        r = subprocess.run([sys.executable, "-m", "moshi_b200.cli", "generate", "--model", str(tmp_path / "m"), "--dtype", dtype,
                            "--prompt", ",".join(map(str, b)), "--max-new", "5"], capture_output=True, text=True, timeout=600, cwd=ROOT)
        assert r.returncode == 0, r.stderr[-2000:]
        got = json.loads(r.stdout.strip().splitlines()[-1])["tokens"]
        want, gaps = orc.greedy(b, 5)
        for g, w, gap in zip(got, want, gaps):
            if g != w:
                assert gap < 1e-3
                break


def drawn_cfg(seed, small):
    """A configuration drawn from the design's space: layer order, head counts and sizes, chunks, rotation, sources of keys and values,
    experts, groups; at toy sizes, or at a small model's layer sizes."""
    g = torch.Generator().manual_seed(seed)

    def pick(*xs):
        return xs[int(torch.randint(0, len(xs), (1,), generator=g))]
    layers = []
    for i in range(pick(2, 3, 4)):
        kind = pick("dense", "moe", "moe", None)
        mlp = None
        if kind == "dense":
            mlp = dense(pick(256, 320, 200) if small else pick(12, 33, 40), limit=pick(0.5, 1.0, 4.0))
        elif kind == "moe":
            n, per = pick(1, 2, 3, 4), pick(3, 4, 5)
            keep = pick(*range(1, n + 1))
            ident = pick(0, 1, 2)
            mlp = moe(n * per - ident, pick(1, 2, 3), pick(64, 96, 40) if small else pick(8, 17, 24), identity=ident, groups=(n, keep) if n > 1 else None,
                      shared=pick(None, 96, 72) if small else pick(None, 11, 16))
        own = [j for j, L in enumerate(layers) if "kv_from" not in L["mixer"]]
        if own and pick(0, 1):
            j = pick(*own)
            L = copy.deepcopy(layers[j])
            L["mixer"].update(kv_from=j, diff=pick(0.2, 0.6, 0.8), scale=L["mixer"]["scale"] * pick(0.8, 1.3))
            L["mixer"].pop("mask", None)
            if pick(0, 1):
                L["mixer"]["mask"] = {"size": pick(50, 64, 100) if small else pick(3, 16, 31)}
            L["mlp"] = mlp
            layers.append(L)
            continue
        kv, dim = pick(1, 2, 3), pick(32, 64, 48, 24) if small else pick(4, 6, 16)
        layers.append(attention(kv * pick(1, 2, 3), kv, dim, pick(32, 64, 96, 40) if small else pick(4, 7, 16), dim ** -0.5 * pick(0.8, 1.4),
                                chunk=pick(0, 48, 130, 256) if small else pick(0, 1, 5, 31, 70), diff=pick(0.2, 0.5, 0.75), rot_dims=pick(0, 2, dim), base=pick(100.0, 1e4, 5e5),
                                factor=pick(None, 2.0, 8.0), mlp=mlp))
    return make_cfg(layers, vocab=pick(320, 777) if small else pick(40, 80), width=pick(128, 160, 200, 256) if small else pick(24, 32, 50), emb=pick(0.5, 1.0, 3.0),
                    eps=pick(1e-5, 1e-6))


@pytest.mark.parametrize("seed", range(8))
def test_configurations_drawn_from_the_designs_space(seed):
    cfg = drawn_cfg(100 + seed, False)
    toks = tokens(80, cfg.vocab, seed)
    for dtype in (torch.float32, torch.bfloat16):
        model, orc = build(cfg, dtype, seed=seed)
        want = orc.forward(toks)
        with gen_for(model) as gen:
            assert_close(gen.step([(0, toks)], list(range(80))), want, dtype, "whole")
            assert_close(in_portions(gen, 1, toks, [37] + [1] * 20 + [2, 5, 2]), want, dtype, "portions")
            assert gen.error_flags() == 0


@pytest.mark.parametrize("seed", range(4))
def test_drawn_models_at_a_small_models_sizes(seed):
    """Whole prompt, prompt + single tokens, and ragged portions with tile-sized and two-token pieces, in both precisions."""
    cfg = drawn_cfg(40 + seed, True)
    toks = tokens(330, cfg.vocab, 60 + seed)
    for dtype in (torch.float32, torch.bfloat16):
        model, orc = build(cfg, dtype, seed=seed)
        want = orc.forward(toks)
        with gen_for(model, capacity=340, max_step_tokens=340) as gen:
            assert_close(gen.step([(0, toks)], list(range(330))), want, dtype, "whole")
            assert_close(in_portions(gen, 1, toks, [290] + [1] * 40), want, dtype, "prompt and single tokens")
            gen.release(1)
            assert_close(in_portions(gen, 1, toks, [2, 3, 17, 97, 2, 33, 64, 5, 31, 2, 16] + [1] * 20), want, dtype, "portions")
            assert gen.error_flags() == 0
