"""The Korirax decoder LM on the GPU against its float64 oracle (``oracle/korirax.py``): every mechanism alone, whole prompts with the
output of every layer run, prompts in portions down to two tokens, token-by-token decoding, unequal batches, slots given back and
used again, distance buckets and query temperatures at their edges, far keys, recurrences with long memories, layers that run
several times, the per-layer token input, the router's groups and correction, the first tokens of a sequence, odd and aligned
sizes, and greedy generation through the scheduler and the command line."""
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
from oracle.korirax import Oracle, layer_runs

from .test_gpu_zz_decoder_lm import gen_for, tokens, write_model
from .test_gpu_zzzzzz_megolorn import TOL, assert_close, in_portions, sharpen

pytestmark = pytest.mark.gpu
ROOT = Path(__file__).resolve().parent.parent
BOTH = pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
RAMP = {"factor": 4.0, "fast": 16.0, "original": 128, "slow": 1.0}


def latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, scale, base=1e4, scaling=None, mlp=None):
    rot = {"base": base, "dims": rot_dim}
    if scaling:
        rot["scaling"] = dict(scaling)
    return {"type": "latent_attention", "mlp": mlp, "mixer": {"dim": dim, "heads": heads, "kv_rank": kv_rank, "q_rank": q_rank, "rot": rot, "rot_dim": rot_dim, "scale": scale, "vdim": vdim}}


def attention(heads, kv, dim, vdim, scale, far=50, buckets=32, temp=None, mlp=None):
    m = {"bias_max": far, "bias_buckets": buckets, "dim": dim, "heads": heads, "kv_heads": kv, "scale": scale, "vdim": vdim}
    if temp:
        m["q_temp"] = {"coef": temp[0], "every": temp[1]}
    return {"type": "attention", "mixer": m, "mlp": mlp}


def rglru(width, blocks, conv, mlp=None):
    return {"type": "rglru", "mixer": {"blocks": blocks, "conv": conv, "width": width}, "mlp": mlp}


def dense(ff):
    return {"ff": ff, "kind": "dense"}


def moe(experts, top, ff, groups=None, shared=None, scale=1.0):
    r = {"experts": experts, "scale": scale, "top": top}
    if groups:
        r["groups"] = {"count": groups[0], "keep": groups[1]}
    d = {"expert": {"ff": ff}, "kind": "moe", "router": r}
    if shared:
        d["shared"] = {"ff": shared}
    return d


def make_cfg(layers, vocab, width, emb=1.5, eps=1e-5, side=0, loop=None):
    d = {"architecture": "Korirax", "embedding": {"scale": emb}, "layers": layers, "norm": {"eps": eps}, "vocab": vocab, "width": width}
    if side:
        d["token_side"] = {"dim": side}
    if loop:
        d["loop"] = {"start": loop[0], "stop": loop[1], "times": loop[2]}
    return DecoderLMConfig.from_dict(d)


# odd sizes: nothing is a multiple of 8; query heads that share key heads and not; value sizes unlike key sizes; ranks, tables and
# convolutions of several sizes; layers in front of, inside and behind the loop; a layer without feed-forward
ODD = make_cfg([rglru(30, 3, 3, mlp=dense(21)),
                attention(6, 2, 10, 12, 0.3, far=23, buckets=10, temp=(0.4, 7), mlp=moe(6, 2, 24, groups=(3, 2), shared=19, scale=1.6)),
                latent(3, 10, 6, 5, 13, 11, 0.25, base=300.0, scaling=RAMP, mlp=moe(5, 2, 17, scale=0.7)),
                rglru(22, 1, 4, mlp=moe(4, 1, 13, groups=(2, 1), shared=9)),
                attention(3, 3, 7, 9, 0.35, far=60, buckets=16, mlp=None),
                latent(5, 6, 2, 7, 9, 20, 0.4, mlp=dense(30))], vocab=97, width=52, side=5, loop=(1, 4, 3))
# aligned sizes: in bfloat16 the linears take the tcgen05 GEMM, attentions, gates and experts their tensor-core kernels
ALIGNED = make_cfg([latent(4, 48, 16, 32, 96, 64, 0.13, base=1e5, scaling=RAMP, mlp=moe(6, 3, 48, groups=(2, 1), shared=64, scale=2.0)),
                    attention(8, 2, 32, 48, 0.18, far=90, temp=(0.25, 16), mlp=dense(128)),
                    rglru(128, 4, 4, mlp=moe(8, 2, 32, groups=(4, 2), shared=32)),
                    attention(4, 4, 64, 80, 0.12, far=40, buckets=24, mlp=None)], vocab=200, width=96, side=16, loop=(0, 3, 2))


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


def moves(a, b, dtype=torch.float32, by=50):
    assert float(logit_error(a, b).max()) > by * TOL[dtype]


@BOTH
@pytest.mark.parametrize("cfg", [ODD, ALIGNED], ids=["odd", "aligned"])
def test_whole_prompt_and_every_layer_run(cfg, dtype):
    model, orc = build(cfg, dtype)
    toks = tokens(90, cfg.vocab, 1)
    want, layers = orc.forward(toks, return_layers=True)
    with gen_for(model, trace_layers=True) as gen:
        got = gen.step([(1, toks)], list(range(len(toks))))
        lo = gen.layer_outputs().cpu()
        assert gen.error_flags() == 0
    assert lo.shape[0] == len(layer_runs(cfg.to_dict())) == layers.shape[0]
    scale = float(layers.abs().max())
    for i in range(layers.shape[0]):
        err = ((lo[i].double() - layers[i]).abs().amax(-1) / scale)
        if dtype == torch.float32:
            assert float(err.max()) < 2e-5, f"run {i}: {float(err.max()):.3g}"
        else:
            assert int((err > 8e-2).sum()) <= 9 and float(err.median()) < 3e-2, f"run {i}: {err.tolist()}"
    assert_close(got, want, dtype)


TINY = dict(blocks=1, conv=1)
ALONE = {
    "latent": [latent(4, 10, 6, 9, 14, 12, 0.3, base=100.0)],
    "latent_ramp": [latent(3, 8, 8, 8, 16, 24, 0.25, scaling=RAMP)],
    "latent_one_head": [latent(1, 5, 2, 3, 7, 3, 0.5)],
    "latent_one_pair_small_rank": [latent(2, 1, 2, 1, 2, 1, 0.7)],
    "latent_factor_one": [latent(2, 8, 4, 8, 8, 8, 0.4, scaling={"factor": 1.0, "fast": 8.0, "original": 64, "slow": 1.0})],
    "latent_wide_rank": [latent(2, 12, 6, 10, 70, 33, 0.2)],
    "attention": [attention(6, 2, 10, 12, 0.3, far=20, buckets=10, temp=(0.3, 9))],
    "attention_no_temperature": [attention(4, 1, 8, 6, 0.3)],
    "attention_own_key_heads": [attention(3, 3, 9, 9, 0.35, far=33, buckets=14, temp=(1.5, 1))],
    "attention_one_head": [attention(1, 1, 16, 4, 0.3, far=500, buckets=6)],
    "attention_two_rows": [attention(2, 1, 6, 6, 0.4, far=9, buckets=2)],
    "attention_many_heads_per_key_head": [attention(20, 1, 6, 5, 0.4, far=15, buckets=12, temp=(0.2, 50))],
    "attention_odd_table": [attention(2, 2, 6, 6, 0.4, far=25, buckets=9)],
    "rglru": [rglru(24, 3, 4)],
    "rglru_one_block": [rglru(19, 1, 2)],
    "rglru_one_tap": [rglru(20, 4, 1)],
    "rglru_six_taps": [rglru(12, 2, 6)],
    "rglru_blocks_of_one": [rglru(7, 7, 3)],
    "rglru_wide": [rglru(96, 2, 5)],
    "dense": [rglru(2, **TINY, mlp=dense(45))],
    "experts": [rglru(2, **TINY, mlp=moe(6, 2, 33))],
    "experts_all_chosen": [rglru(2, **TINY, mlp=moe(3, 3, 20, scale=3.0))],
    "experts_top_one": [rglru(2, **TINY, mlp=moe(8, 1, 20, groups=(4, 1), shared=31))],
    "experts_groups_of_one": [rglru(2, **TINY, mlp=moe(5, 2, 20, groups=(5, 3)))],
    "experts_all_groups_kept": [rglru(2, **TINY, mlp=moe(8, 4, 16, groups=(4, 4), shared=16, scale=0.5))],
    "experts_sixty": [rglru(2, **TINY, mlp=moe(60, 6, 9, groups=(6, 3), shared=5))],
}


@pytest.mark.parametrize("side", [0, 7], ids=["plain", "side"])
@pytest.mark.parametrize("what", sorted(ALONE))
def test_mechanisms_in_isolation(what, side):
    cfg = make_cfg(copy.deepcopy(ALONE[what]), vocab=61, width=44, emb=0.7, side=side)
    model, orc = build(cfg, torch.float32, seed=11)
    toks = tokens(70, cfg.vocab, 2)
    want = orc.forward(toks)
    with gen_for(model) as gen:
        assert_close(gen.step([(0, toks)], list(range(len(toks)))), want, torch.float32, what)
        assert_close(in_portions(gen, 1, toks, [41, 2] + [1] * 20), want, torch.float32, what + ", portions")


@BOTH
@pytest.mark.parametrize("buckets,far", [(32, 100), (8, 40), (6, 64), (20, 131), (4, 5), (12, 7)])
def test_bias_buckets_at_their_edges(buckets, far, dtype):
    """Large table entries of alternating sign, so that a distance in the wrong bucket shows; the oracle itself moves by far more than
    the tolerance when an edge moves by one.  bfloat16 takes the tensor-core kernels, with the table in shared memory."""
    by = 4.0 if dtype == torch.float32 else 2.0
    cfg = make_cfg([attention(4, 2, 16, 16, 0.3, far=far, buckets=buckets)], vocab=53, width=48)

    def edit(t):
        rel = t["l0.mix.rel"]
        sign = 1.0 - 2.0 * (torch.arange(rel.shape[0]) % 2)
        t["l0.mix.rel"] = (by * sign[:, None] * (0.5 + rel.float().abs())).to(rel.dtype)
    model, orc = build(cfg, dtype, seed=5, edit=edit)
    n = max(150, far + 60)
    toks = tokens(n, cfg.vocab, 3)
    want = orc.forward(toks)
    moved = cfg.to_dict()
    moved["layers"][0]["mixer"]["bias_max"] = far * 1.5 + 1
    moves(Oracle(moved, orc.t).forward(toks), want, dtype, 20 if dtype == torch.float32 else 1.5)
    with gen_for(model, capacity=n + 8, max_step_tokens=max(256, n)) as gen:
        def close(got, what):
            e = logit_error(got.cpu(), want)
            assert float(e.max()) < TOL[dtype], f"{what}: {float(e.max()):.3g} at {int(e.argmax())}"
        close(gen.step([(0, toks)], list(range(n))), "whole")
        gen.release(0)
        close(in_portions(gen, 0, toks, [far + 1, 2, 3] + [1] * 40 + [2] * 5), "portions and single tokens")
        for split in (2, 5):
            gen.release(0)
            gen.set_option("attn_split", split)
            close(in_portions(gen, 0, toks, [n - 30] + [1] * 30), f"keys cut {split} times")
        gen.set_option("attn_split", 0)


@pytest.mark.parametrize("every", [1, 3, 16, 64])
def test_query_temperature_at_its_steps(every):
    cfg = make_cfg([attention(4, 2, 12, 8, 0.4, temp=(0.8, every))], vocab=53, width=40)
    model, orc = build(cfg, torch.float32, seed=8, edit=sharpen(2.0))
    toks = tokens(140, cfg.vocab, 4)
    want = orc.forward(toks)
    d = cfg.to_dict()
    d["layers"][0]["mixer"]["q_temp"]["every"] = every + 1
    moves(Oracle(d, orc.t).forward(toks), want)
    with gen_for(model) as gen:
        assert_close(gen.step([(0, toks)], list(range(140))), want, torch.float32, "whole")
        assert_close(in_portions(gen, 1, toks, [every, 2] + [1] * 70), want, torch.float32, "portions and single tokens")


def sharpen_latent(by):
    """The latents are normed, so their norms' weights set how sharp the scores are."""
    def edit(t):
        for k in t:
            if k.endswith("dq.norm"):
                t[k] = t[k] * by
    return edit


@BOTH
@pytest.mark.parametrize("kind", ["attention", "latent", "latent_aligned"])
def test_a_far_key(kind, dtype):
    """Sharp scores over 600 tokens, so that single keys hundreds of positions back carry rows of the result: in a prompt, in portions
    and in single tokens."""
    layer = {"attention": attention(4, 2, 16, 16, 0.5, far=30), "latent": latent(4, 12, 4, 16, 24, 20, 0.5, scaling=RAMP),
             "latent_aligned": latent(4, 48, 16, 32, 112, 64, 0.22, base=1e5)}[kind]
    cfg = make_cfg([layer], vocab=53, width=48)
    by = 2.0 if dtype == torch.float32 else 1.3
    model, orc = build(cfg, dtype, seed=6, edit=sharpen(by) if kind == "attention" else sharpen_latent(by * by))
    toks = tokens(600, cfg.vocab, 5)
    want = orc.forward(toks)
    short = orc.forward(toks[300:])                   # the same last tokens without the first 300: the far keys matter
    moves(short[-40:], want[-40:])
    with gen_for(model, capacity=640, max_step_tokens=640) as gen:
        assert_close(gen.step([(0, toks)], list(range(600))), want, dtype, "whole")
        gen.release(0)
        assert_close(in_portions(gen, 0, toks, [517, 2, 33] + [1] * 40), want, dtype, "portions and single tokens")
        for split in (2, 7):
            gen.release(0)
            gen.set_option("attn_split", split)
            assert_close(in_portions(gen, 0, toks, [590] + [1] * 10), want, dtype, f"keys cut {split} times")
        gen.set_option("attn_split", 0)
        assert gen.error_flags() == 0


@pytest.mark.parametrize("heads,kv,dim,vdim,far", [(4, 2, 16, 16, 40), (8, 8, 32, 64, 100), (6, 2, 48, 112, 20), (20, 1, 16, 32, 120), (20, 1, 16, 32, 600), (70, 1, 16, 16, 30),
                                                   (3, 1, 128, 128, 60), (2, 1, 64, 144, 60), (2, 2, 32, 256, 25), (2, 1, 16, 272, 25), (4, 2, 24, 40, 60), (3, 3, 112, 96, 70)])
def test_both_attention_kernels_in_bfloat16(heads, kv, dim, vdim, far):
    """Tensor cores and CUDA cores on the same bf16 cache: prompts, single tokens, keys cut over CTAs, tiles that cut a token's heads
    (20 and 70 query heads per key head), value sizes up to 256 columns and beyond, a bias table that stays in global memory, and
    sizes that only the CUDA cores take."""
    cfg = make_cfg([attention(heads, kv, dim, vdim, dim ** -0.5, far=far, temp=(0.3, 40))], vocab=53, width=64)
    model, orc = build(cfg, torch.bfloat16, seed=7, edit=sharpen(1.3))
    toks = tokens(150, cfg.vocab, 9)
    want = orc.forward(toks)
    with gen_for(model) as gen:
        for tc in (1, 0):
            gen.set_option("attn_tc", tc)
            for split in (0, 1, 3):
                gen.set_option("attn_split", split)
                gen.release(0)
                e = logit_error(in_portions(gen, 0, toks, [101, 17] + [1] * 25).cpu(), want)
                assert float(e.max()) < TOL[torch.bfloat16], f"attn_tc {tc}, attn_split {split}: {float(e.max()):.3g} at {int(e.argmax())}"
        assert gen.error_flags() == 0


@pytest.mark.parametrize("heads,dim,rot_dim,vdim,kv_rank,q_rank", [(4, 48, 16, 64, 112, 80), (3, 16, 8, 16, 56, 40), (2, 24, 8, 8, 40, 10), (16, 64, 64, 64, 512, 96), (2, 16, 2, 16, 30, 16),
                                                                    (24, 16, 16, 16, 48, 7)])
def test_latent_attention_sizes_in_bfloat16(heads, dim, rot_dim, vdim, kv_rank, q_rank):
    cfg = make_cfg([latent(heads, dim, rot_dim, vdim, kv_rank, q_rank, (dim + rot_dim) ** -0.5, scaling=RAMP)], vocab=53, width=64)
    model, orc = build(cfg, torch.bfloat16, seed=7, edit=sharpen_latent(1.3))
    toks = tokens(150, cfg.vocab, 9)
    want = orc.forward(toks)
    with gen_for(model) as gen:
        for tc in (1, 0):
            gen.set_option("attn_tc", tc)
            for split in (0, 3):
                gen.set_option("attn_split", split)
                gen.release(0)
                e = logit_error(in_portions(gen, 0, toks, [101, 17] + [1] * 25).cpu(), want)
                assert float(e.max()) < TOL[torch.bfloat16], f"attn_tc {tc}, attn_split {split}: {float(e.max()):.3g} at {int(e.argmax())}"
        assert gen.error_flags() == 0


@BOTH
@pytest.mark.parametrize("width,blocks,conv", [(48, 3, 4), (33, 3, 2), (256, 2, 4), (40, 5, 8)])
def test_recurrence_with_a_long_memory(width, blocks, conv, dtype):
    """Decays next to one: token 0 still moves the logits 300 tokens later.  Portions shorter than the convolution, segments of every
    count, single tokens, and two requests of different lengths in one step."""
    cfg = make_cfg([rglru(width, blocks, conv)], vocab=53, width=40)

    def edit(t):
        t["l0.mix.lam"] = torch.full_like(t["l0.mix.lam"], -8.5)
    model, orc = build(cfg, dtype, seed=9, edit=edit)
    toks = tokens(420, cfg.vocab, 6)
    want = orc.forward(toks)
    other = orc.forward([(toks[0] + 1) % 53] + toks[1:])
    moves(other[300:320], want[300:320], by=20)
    b = tokens(37, cfg.vocab, 7)
    wb = orc.forward(b)
    with gen_for(model, capacity=480, max_step_tokens=480) as gen:
        for tc in (1, 0):
            gen.set_option("attn_tc", tc)
            gen.release(0)
            assert_close(gen.step([(0, toks)], list(range(420))), want, dtype, "whole")
            gen.release(0)
            assert_close(in_portions(gen, 0, toks, [3, 1, 2, 2, 17, 33, 130, 64, 2] + [1] * 40), want, dtype, "portions and single tokens")
            gen.release(0)
            gen.release(1)
            gen.step([(0, toks[:300]), (1, b[:5])], [])
            got = gen.step([(1, b[5:6]), (0, toks[300:])], list(range(121)))
            assert_close(got[:1], wb[5:6], dtype, "one token beside a portion")
            assert_close(got[1:], want[300:], dtype, "a portion beside one token")
            got = gen.step([(1, b[6:])], list(range(31)))
            assert_close(got, wb[6:], dtype, "its next portion")


@BOTH
@pytest.mark.parametrize("conv", [1, 4, 7, 12])
def test_convolution_in_steps_of_many_tokens(conv, dtype):
    """Steps of at least 512 tokens take the convolution on tiles of eight tokens: one prompt, then requests of several lengths on
    several histories whose borders cut the tiles, single tokens among them."""
    cfg = make_cfg([rglru(36, 3, conv, mlp=dense(24)), rglru(32, 2, conv)], vocab=53, width=40, side=4)
    model, orc = build(cfg, dtype, seed=19)
    a, b, c, d = tokens(1060, cfg.vocab, 8), tokens(13, cfg.vocab, 9), tokens(4, cfg.vocab, 10), tokens(60, cfg.vocab, 11)
    wa, wb, wc, wd = (orc.forward(x) for x in (a, b, c, d))
    with gen_for(model, slots=4, capacity=1100, max_step_tokens=700) as gen:
        assert_close(gen.step([(0, a[:519])], list(range(519))), wa[:519], dtype, "one prompt")
        gen.step([(1, b[:12]), (3, d[:2])], [])
        got = gen.step([(1, b[12:]), (3, d[2:]), (2, c), (0, a[519:])], list(range(1 + 58 + 4 + 541)))
        for lo, w, what in ((0, wb[12:], "b"), (1, wd[2:], "d"), (59, wc, "c"), (63, wa[519:], "a")):
            assert_close(got[lo:lo + len(w)], w, dtype, what)


@pytest.mark.parametrize("loop", [(0, 1, 1), (0, 2, 2), (1, 2, 4), (0, 3, 2), (1, 3, 3), (2, 3, 2)])
def test_loops_anywhere_with_a_cache_per_pass(loop):
    layers = [attention(2, 1, 8, 6, 0.4, far=20, buckets=8, mlp=dense(20)), rglru(18, 2, 3, mlp=moe(4, 2, 12)), latent(2, 6, 4, 5, 10, 8, 0.4)]
    for side in (0, 6):
        cfg = make_cfg(copy.deepcopy(layers), vocab=53, width=40, side=side, loop=loop)
        model, orc = build(cfg, torch.float32, seed=12)
        toks = tokens(75, cfg.vocab, 7)
        want, lw = orc.forward(toks, return_layers=True)
        still = dict(orc.t)
        still["loop.step"] = torch.zeros_like(still["loop.step"])
        moves(Oracle(cfg.to_dict(), still).forward(toks), want)
        with gen_for(model, trace_layers=True) as gen:
            assert_close(gen.step([(0, toks)], list(range(75))), want, torch.float32, "whole")
            lo = gen.layer_outputs().cpu()
            assert float((lo.double() - lw).abs().max()) < 3e-5 * float(lw.abs().max())
            assert_close(in_portions(gen, 1, toks, [31, 2, 5] + [1] * 20), want, torch.float32, "portions")


@pytest.mark.parametrize("side", [3, 8, 24, 100])
def test_token_input_for_few_and_many_tokens(side):
    """Up to 64 tokens take the one-launch gate product, more the GEMM: both, in both precisions; the oracle moves when the layers'
    parts of the second table are exchanged."""
    cfg = make_cfg([rglru(16, 1, 2, mlp=dense(24)), attention(2, 1, 16, 16, 0.3), rglru(16, 2, 2)], vocab=53, width=64, side=side)
    toks = tokens(150, cfg.vocab, 8)
    for dtype in (torch.float32, torch.bfloat16):
        model, orc = build(cfg, dtype, seed=13)
        want = orc.forward(toks)
        other = dict(orc.t)
        other["side.embed"] = other["side.embed"].view(53, 3, side).flip(1).reshape(53, -1)
        moves(Oracle(cfg.to_dict(), other).forward(toks), want, dtype, 2)
        with gen_for(model) as gen:
            assert_close(gen.step([(0, toks)], list(range(150))), want, dtype, "whole")
            assert_close(in_portions(gen, 1, toks, [65, 64, 2] + [1] * 10), want, dtype, "portions")


def test_router_with_negative_choice_scores_and_groups_by_two():
    """All choice scores negative (the groups that are left out must not win with a zero), corrections as large as the scores; the
    oracle moves when the correction or the groups are left out, and when a group is judged by its best score alone."""
    cfg = make_cfg([rglru(8, 1, 2, mlp=moe(12, 3, 25, groups=(4, 2), shared=10, scale=1.8))] * 2, vocab=61, width=44)

    def edit(t):
        for k in t:
            if k.endswith("correction"):
                t[k] = (torch.linspace(-1.9, -1.5, t[k].numel()) - 0.3 * (torch.arange(t[k].numel()) % 3 == 1)).to(t[k].dtype)
            if k.endswith("router"):
                t[k] = t[k] * 3.0
    model, orc = build(cfg, torch.float32, seed=17, edit=edit)
    toks = tokens(120, cfg.vocab, 16)
    want = orc.forward(toks)
    flat = dict(orc.t)
    for k in flat:
        if k.endswith("correction"):
            flat[k] = torch.zeros_like(flat[k])
    moves(Oracle(cfg.to_dict(), flat).forward(toks), want)
    for groups in (None, {"count": 12, "keep": 6}):
        d = cfg.to_dict()
        for L in d["layers"]:
            L["mlp"]["router"].pop("groups")
            if groups:
                L["mlp"]["router"]["groups"] = groups
        moves(Oracle(d, orc.t).forward(toks), want)
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


@BOTH
def test_slots_are_given_back_and_used_again(dtype):
    cfg = ODD if dtype == torch.float32 else ALIGNED
    model, orc = build(cfg, dtype)
    a, b = tokens(120, cfg.vocab, 12), tokens(11, cfg.vocab, 13)
    wa, wb = orc.forward(a), orc.forward(b)
    with gen_for(model, slots=1) as gen:
        gen.step([(0, a)], [])
        with pytest.raises(RuntimeError):
            gen.step([(0, tokens(200, cfg.vocab, 14))], [])                                 # would overflow the slot: refused whole
        for cuts in ([], [1] * 11, [2, 1]):
            gen.release(0)
            assert gen.slot_length(0) == 0
            assert_close(in_portions(gen, 0, b, cuts), wb, dtype, f"reused, {cuts}")
        gen.release(0)
        assert_close(in_portions(gen, 0, a, [3, 50]), wa, dtype, "again")


def test_configurations_that_the_handle_refuses():
    from moshi_b200.models import DecoderLM
    for L in (attention(3, 2, 8, 8, 0.3), latent(2, 8, 3, 8, 8, 8, 0.3), latent(2, 8, 4, 8, 1024, 8, 0.3), rglru(8, 2, 0), attention(2, 1, 8, 8, 0.3, mlp=moe(5, 2, 8, groups=(2, 1))),
              attention(2, 1, 8, 8, 0.3, mlp=moe(6, 3, 8, groups=(3, 1))), attention(2, 1, 8, 8, 0.3, far=0), attention(2, 1, 8, 8, 0.3, mlp=dense(0))):
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
    """A configuration drawn from the design's space: layer order, head counts and sizes, ranks, tables, temperatures, taps, blocks,
    experts, groups, loop, token input; at toy sizes, or at a small model's layer sizes."""
    g = torch.Generator().manual_seed(seed)

    def pick(*xs):
        return xs[int(torch.randint(0, len(xs), (1,), generator=g))]
    layers = []
    for i in range(pick(2, 3, 4)):
        kind = pick("dense", "moe", "moe", None)
        mlp = None
        if kind == "dense":
            mlp = dense(pick(256, 320, 200) if small else pick(12, 33, 40))
        elif kind == "moe":
            n, per = pick(1, 2, 3, 4), pick(3, 4, 5)
            mlp = moe(n * per, pick(1, 2, 3), pick(64, 96, 40) if small else pick(8, 17, 24), groups=(n, pick(*range(1, n + 1))) if n > 1 else None,
                      shared=pick(None, 96, 72) if small else pick(None, 11, 16), scale=pick(1.0, 0.5, 2.2))
        t = pick("latent", "attention", "rglru")
        if t == "latent":
            dim, rd = (pick(32, 64, 24), pick(8, 16, 32)) if small else (pick(4, 7, 16), pick(2, 4, 6))
            layers.append(latent(pick(1, 3, 4, 6), dim, rd, pick(32, 48, 20) if small else pick(3, 8, 10), pick(64, 112, 96, 50) if small else pick(5, 16, 21),
                                 pick(64, 72, 48, 30) if small else pick(4, 9, 16), (dim + rd) ** -0.5 * pick(0.8, 1.4), base=pick(100.0, 1e4, 5e5),
                                 scaling=pick(None, RAMP, {"factor": 16.0, "fast": 32.0, "original": 300, "slow": 2.0}), mlp=mlp))
        elif t == "attention":
            kv, dim, B = pick(1, 2, 3), pick(32, 64, 48, 24) if small else pick(4, 6, 16), pick(8, 16, 32)
            layers.append(attention(kv * pick(1, 2, 3), kv, dim, pick(32, 64, 96, 40) if small else pick(4, 7, 16), dim ** -0.5 * pick(0.8, 1.4),
                                    far=pick(B // 2 + 1, 60, 200), buckets=B, temp=pick(None, (0.3, 10), (0.1, 100)), mlp=mlp))
        else:
            nb = pick(1, 2, 3)
            layers.append(rglru(nb * (pick(32, 48, 20, 64) if small else pick(1, 5, 8)), nb, pick(1, 2, 4, 5), mlp=mlp))
    n = len(layers)
    start = pick(*range(n))
    loop = pick(None, (start, pick(*range(start + 1, n + 1)), pick(1, 2, 3)))
    return make_cfg(layers, vocab=pick(320, 777) if small else pick(40, 80), width=pick(128, 160, 200, 256) if small else pick(24, 32, 50), emb=pick(0.5, 1.0, 3.0),
                    eps=pick(1e-5, 1e-6), side=pick(0, 16, 30) if small else pick(0, 3, 8), loop=loop)


@pytest.mark.parametrize("seed", range(10))
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


@pytest.mark.parametrize("seed", range(6))
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
