"""Rikolix through the engine against the plain implementation (tests/plain/rikolix_plain.py): configuration and the
oracle's own mechanisms on the CPU; on a GPU each kernel against its formula, each mechanism alone, prompts against
token-by-token decoding, portions down to two tokens, mixed batches with pages and slots used again, sharpened scores that
show a lost far key, long decoding, and greedy generation through the public entry point."""
import copy
import json
import math
import os
import random
import subprocess
import sys
import types

import pytest
import torch

import helpers
from plain import rikolix_plain as plain

TOL = {"float32": helpers.TOL["float32"], "bfloat16": 2.0 * helpers.TOL["bfloat16"]}      # bfloat16: every sublayer's output is normed, rounding included


def latent(heads, dim, rot_dim, vdim, q_rank, kv_rank, base=100.0, scale=None, kv_from=None):
    m = dict(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, q_rank=q_rank, kv_rank=kv_rank, rot=dict(base=base, dims=rot_dim),
             scale=scale or 1.0 / math.sqrt(dim + rot_dim))
    if kv_from is not None:
        m["kv_from"] = kv_from
    return dict(type="latent_attention", mixer=m)


def attention(heads, kv_heads, dim, vdim, dims, base=1000.0, scale=None):
    return dict(type="attention", mixer=dict(heads=heads, kv_heads=kv_heads, dim=dim, vdim=vdim, rot=dict(base=base, dims=dims),
                                             scale=scale or 1.0 / math.sqrt(dim)))


def dense(ff):
    return dict(kind="dense", ff=ff)


def moe(experts, top, ff, identity=0, groups=None):
    router = dict(experts=experts, top=top, identity=identity)
    if groups is not None:
        router["groups"] = dict(count=groups[0], keep=groups[1])
    return dict(kind="moe", expert=dict(ff=ff), router=router)


def layer(mixer, mlp=None):
    return dict(mixer, mlp=mlp)


def config(layers, vocab, width, eps=1e-5, scale=1.0):
    return dict(architecture="Rikolix", vocab=vocab, width=width, norm=dict(eps=eps), embedding=dict(scale=scale), layers=layers)


# Every size differs between the configurations and within them: query latents wider and narrower than the key latent, plain,
# rotated and value parts of different widths, borrowed rows under other head counts and value widths than the owner's, two
# owners with a borrower each, groups of one, two and three query heads, a whole head that turns and a part of one, values
# wider and narrower than the keys, routers with and without groups and identity outputs, one group of one, one expert of one,
# all outputs chosen, layers without a feed-forward, an embedding scale of one.
RIKO_A = config([
    layer(latent(3, 12, 6, 10, 28, 20), dense(56)),
    layer(attention(4, 2, 16, 24, 8), moe(5, 2, 24, identity=1, groups=(3, 2))),
    layer(latent(2, 8, 6, 16, 12, 20, kv_from=0), moe(3, 2, 16, identity=3, groups=(2, 1))),
    layer(latent(4, 6, 4, 8, 16, 12, base=30.0)),
    layer(latent(5, 10, 4, 6, 40, 12, base=30.0, kv_from=3), dense(40)),
    layer(attention(3, 3, 8, 8, 8, base=300.0), moe(4, 1, 32)),
], vocab=180, width=48, scale=0.7)
RIKO_B = config([
    layer(attention(6, 2, 12, 20, 4, base=50.0), moe(1, 1, 48)),
    layer(latent(5, 8, 8, 12, 20, 24, base=500.0), moe(6, 3, 16, identity=2, groups=(4, 4))),
    layer(attention(2, 1, 32, 16, 32)),
    layer(latent(1, 16, 2, 16, 8, 24, base=20.0), moe(2, 4, 24, identity=2)),
], vocab=131, width=40, eps=3e-6, scale=2.5)
# head sizes at which the bfloat16 engine's prompt attention runs on the tensor cores, widths its fused products take
RIKO_C = config([
    layer(latent(2, 128, 64, 128, 96, 80, base=10000.0), dense(160)),
    layer(attention(6, 2, 64, 64, 32, base=10000.0), moe(6, 2, 32, identity=2, groups=(2, 1))),
    layer(latent(3, 128, 64, 128, 64, 80, base=10000.0, kv_from=0), moe(4, 2, 64, identity=2)),
    layer(attention(2, 1, 128, 128, 128, base=5000.0)),
    layer(attention(2, 2, 64, 128, 64, base=5000.0), dense(96)),
], vocab=150, width=64, eps=1e-6, scale=1.5)
# no routed layer: the bfloat16 engine is held to the bar at every position
RIKO_D = config([
    layer(latent(4, 16, 8, 24, 48, 32, base=1000.0), dense(64)),
    layer(attention(4, 4, 32, 16, 16)),
    layer(latent(2, 32, 8, 8, 16, 32, base=1000.0, kv_from=0), dense(96)),
    layer(attention(2, 1, 64, 64, 64), dense(48)),
], vocab=140, width=56, eps=2e-6)
ALONE = {
    "latent": config([layer(latent(3, 12, 6, 10, 28, 20))], vocab=64, width=40),
    "borrowed": config([layer(latent(2, 8, 4, 8, 8, 12)), layer(latent(3, 6, 4, 10, 16, 12, kv_from=0))], vocab=64, width=40),
    "attention": config([layer(attention(4, 2, 16, 24, 8))], vocab=64, width=40),
    "attention_all_turns": config([layer(attention(3, 1, 8, 8, 8))], vocab=64, width=40, scale=3.0),
    "dense": config([layer(attention(2, 2, 8, 8, 4), dense(48))], vocab=64, width=40),
    "moe": config([layer(latent(2, 8, 4, 8, 8, 8), moe(6, 2, 24))], vocab=64, width=40),
    "moe_groups": config([layer(latent(2, 8, 4, 8, 8, 8), moe(6, 2, 24, groups=(3, 1)))], vocab=64, width=40),
    "moe_identity": config([layer(latent(2, 8, 4, 8, 8, 8), moe(3, 3, 16, identity=3, groups=(2, 2)))], vocab=64, width=40),
}
CONFIGS = {"A": (RIKO_A, 51, 8), "B": (RIKO_B, 52, 4), "C": (RIKO_C, 53, 16), "D": (RIKO_D, 54, 8)}      # config, seed, page size


# ------------------------------------------------------------------ configuration (CPU)
def test_config_becomes_parts():
    from pulsar_b200.config import config_from_dict
    from pulsar_b200.models import build_model
    cfg = config_from_dict(copy.deepcopy(RIKO_A))
    spec = cfg.model_spec()
    assert [(c.block, c.cache) for c in spec.run_order] == [(0, 0), (1, 1), (2, 0), (3, 2), (4, 2), (5, 3)]      # borrowers name the owner's entry
    assert spec.embedding_multiplier == 0.7 and spec.logit_scale == 1.0
    assert all(b.kind == "sandwich" and b.mixer_norm.about_one and b.mixer_post_norm.about_one for b in spec.blocks) and spec.final_norm.about_one
    m0, m1, m2 = (spec.blocks[i].mixer for i in range(3))
    assert (m0.kind, m0.option("q_rank"), m0.option("kv_rank"), m0.option("rot_dim"), m0.head_dim, m0.value_dim, m0.own_kv) == \
        ("latent_attention", 28, 20, 6, 12, 10, True)
    assert not m2.own_kv and (m2.n_heads, m2.value_dim, m2.option("q_rank")) == (2, 16, 12)
    assert (m1.qk_norm_whole, m1.qk_norm_eps, m1.rotate_neighbours, m1.sigmoid_weights, m1.score_bias) == (True, 1e-5, True, True, True)
    assert (m1.position.rotary_dim, m1.position.theta, m1.value_position.rotary_dim, m1.value_position.theta) == (8, 1000.0, 24, 1000.0)
    ff = spec.blocks[1].feed_forward
    assert (ff.option("experts"), ff.option("identity"), ff.option("groups"), ff.option("gated"), ff.option("scoring"), ff.option("renormalize")) == \
        (5, 1, (3, 2), False, "softmax", False)
    assert spec.blocks[0].feed_forward.activation == "relu2" and spec.blocks[3].feed_forward is None
    assert spec.blocks[5].feed_forward.option("groups") is None and spec.blocks[5].feed_forward.option("identity") == 0
    assert cfg.to_dict() == RIKO_A
    model = build_model(cfg, torch.float32)
    shapes = {w.name: tuple(w.shape) for w in model.weight_specs()}
    assert shapes["l0.mix.dq"] == (28, 48) and shapes["l0.mix.dq.norm"] == (28,) and shapes["l0.mix.uq"] == (3 * 18, 28)
    assert shapes["l0.mix.dkv"] == (26, 48) and shapes["l0.mix.dkv.norm"] == (20,) and shapes["l0.mix.uk"] == (36, 20)
    assert shapes["l0.mix.uv"] == (30, 20) and shapes["l0.mix.o"] == (48, 30)
    assert shapes["l2.mix.uk"] == (16, 20) and shapes["l2.mix.uv"] == (32, 20) and "l2.mix.dkv" not in shapes and "l2.mix.dkv.norm" not in shapes
    assert shapes["l1.mix.q"] == (64, 48) and shapes["l1.mix.k"] == (32, 48) and shapes["l1.mix.v"] == (48, 48)
    assert shapes["l1.mix.q.norm"] == (64,) and shapes["l1.mix.k.norm"] == (32,) and shapes["l1.mix.pb"] == (4,) and shapes["l1.mix.o"] == (48, 96)
    assert shapes["l1.mlp.router"] == (6, 48) and shapes["l1.mlp.correction"] == (6,) and "l1.mlp.e5.up" not in shapes
    assert shapes["l1.mlp.e4.up"] == (24, 48) and shapes["l1.mlp.e4.down"] == (48, 24) and "l1.mlp.e0.gate" not in shapes
    assert shapes["l0.mlp.up"] == (56, 48) and "l3.norm2" not in shapes and shapes["l3.norm1b"] == (48,)
    needs = model.cache_needs()
    assert [[(t.name, t.heads, t.width) for t in n.tensors] for n in needs] == [
        [("latent", 1, 26)], [("k", 2, 16), ("v", 2, 24)], [("latent", 1, 16)], [("k", 3, 8), ("v", 3, 8)]]


@pytest.mark.parametrize("edit,match", [
    (lambda c: c["layers"][1]["mixer"].update(kv_heads=3), "multiple"),
    (lambda c: c["layers"][1]["mixer"].update(vdim=7), "even"),
    (lambda c: c["layers"][1]["mixer"]["rot"].update(dims=18), "dims"),
    (lambda c: c["layers"][1]["mixer"].pop("rot"), "rot"),
    (lambda c: c["layers"][0].update(type="mamba1"), "latent_attention"),
    (lambda c: c["layers"][0]["mixer"].pop("q_rank"), "q_rank"),
    (lambda c: c["layers"][0]["mixer"].pop("scale"), "scale"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=1), "no latent"),
    (lambda c: c["layers"][2]["mixer"].update(kv_from=2), "earlier"),
    (lambda c: c["layers"][4]["mixer"].update(kv_from=2), "no latent"),
    (lambda c: c["layers"][2]["mixer"].update(kv_rank=24), "equal"),
    (lambda c: c["layers"][0]["mlp"].update(kind="gated"), "kind"),
    (lambda c: c["layers"][1]["mlp"]["router"].update(top=5), "top"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(count=4), "count"),
    (lambda c: c["layers"][1]["mlp"]["router"]["groups"].update(keep=4), "keep"),
    (lambda c: c["layers"][1]["mlp"].pop("expert"), "expert"),
    (lambda c: c.pop("norm"), "norm"),
])
def test_config_errors(edit, match):
    from pulsar_b200.config import ConfigError, config_from_dict
    raw = copy.deepcopy(RIKO_A)
    edit(raw)
    with pytest.raises(ConfigError, match=match):
        config_from_dict(raw)


def test_parts_refuse_what_they_do_not_compute():
    from pulsar_b200.config.specs import FeedForwardSpec, MixerSpec, PositionSpec
    from pulsar_b200.parts.attention import Attention
    from pulsar_b200.parts.moe import MixtureOfExperts
    base = dict(kind="attention", hidden=16, n_heads=2, n_kv_heads=1, head_dim=8, scale=1.0)
    for more, match in ((dict(score_bias=True), "sigmoid"), (dict(sigmoid_weights=True, sinks=True), "sink"),
                        (dict(qk_norm_whole=True), "eps"), (dict(value_position=PositionSpec("rope", 8, 4, 10.0)), "all their"),
                        (dict(rotate_neighbours=True, output_gate=True), "plain"), (dict(rotate_neighbours=True, qk_norm_eps=1e-5), "per-head")):
        with pytest.raises(ValueError, match=match):
            Attention(MixerSpec(**base, **more), "", torch.float32)
    for more, match in ((dict(gated=False), "relu2"), (dict(identity=1, weight_input=True), "inputs"), (dict(groups=(3, 1)), "groups")):
        with pytest.raises(ValueError, match=match):
            MixtureOfExperts(FeedForwardSpec("moe", 16, 8, "silu", extra=tuple(dict(experts=4, top=2, **more).items())), "", torch.float32)


def test_plain_mechanisms_agree_with_loops_over_single_numbers():
    """The oracle's vectorised forms against the equations written out one token, one head and one pair at a time."""
    g = torch.Generator().manual_seed(3)
    rnd = lambda *shape: torch.randn(*shape, generator=g, dtype=torch.float64)
    L, W, eps = 7, 10, 1e-6
    h = rnd(L, W)
    unit = lambda v: v / math.sqrt(float((v * v).mean()) + eps)

    def turned(v, t, base, dims, sign=1.0):
        v = v.clone()
        for i in range(dims // 2):
            ang = sign * t * base ** (-2.0 * i / dims)
            a, b = float(v[2 * i]), float(v[2 * i + 1])
            v[2 * i], v[2 * i + 1] = a * math.cos(ang) - b * math.sin(ang), b * math.cos(ang) + a * math.sin(ang)
        return v
    assert float((plain.rms_norm_about_one(h, h[0], eps)[3] - unit(h[3]) * (1 + h[0])).abs().max()) < 1e-12
    # sigmoid attention: one query, one head, one key at a time
    m = attention(4, 2, 6, 4, 4, base=10.0, scale=0.4)["mixer"]
    w = {"q": rnd(24, W), "k": rnd(12, W), "v": rnd(8, W), "o": rnd(W, 16), "q.norm": rnd(24), "k.norm": rnd(12), "pb": rnd(4)}
    out = plain.sigmoid_attention(h, w, m, eps)
    for i in range(L):
        heads = []
        q = unit(w["q"] @ h[i]) * w["q.norm"]
        for hd in range(4):
            kv = hd // 2
            acc = torch.zeros(4, dtype=torch.float64)
            for j in range(i + 1):
                k = (unit(w["k"] @ h[j]) * w["k.norm"])[kv * 6:(kv + 1) * 6]
                s = float(turned(q[hd * 6:(hd + 1) * 6], i, 10.0, 4) @ turned(k, j, 10.0, 4)) * 0.4 + float(w["pb"][hd])
                # turned by j, then back by i: by the difference of the two
                acc += turned((w["v"] @ h[j])[kv * 4:(kv + 1) * 4], j - i, 10.0, 4) / (1.0 + math.exp(-s))
            heads.append(acc)
        assert float((w["o"] @ torch.cat(heads) - out[i]).abs().max()) < 1e-10
    # latent attention over its own rows and over borrowed ones
    m = latent(2, 3, 4, 5, 6, 7, base=10.0, scale=0.3)["mixer"]
    w = {"dq": rnd(6, W), "dq.norm": rnd(6), "uq": rnd(14, 6), "dkv": rnd(11, W), "dkv.norm": rnd(7), "uk": rnd(6, 7), "uv": rnd(10, 7),
         "o": rnd(W, 10)}
    own = plain.latent_rows(h, w, m, eps)
    other = (rnd(L, 7), rnd(L, 4))
    for rows in (own, other):
        out = plain.latent_attention(h, w, m, eps, rows)
        for i in (0, 3, 6):
            heads = []
            for hd in range(2):
                q = (w["uq"] @ (unit(w["dq"] @ h[i]) * w["dq.norm"]))[hd * 7:(hd + 1) * 7]
                e = [math.exp(0.3 * (float(q[:3] @ (w["uk"] @ rows[0][j])[hd * 3:(hd + 1) * 3]) +
                                     float(turned(q[3:], i, 10.0, 4) @ rows[1][j]))) for j in range(i + 1)]
                heads.append(sum(x / sum(e) * (w["uv"] @ rows[0][j])[hd * 5:(hd + 1) * 5] for j, x in enumerate(e)))
            assert float((w["o"] @ torch.cat(heads) - out[i]).abs().max()) < 1e-10
    down = w["dkv"] @ h[4]
    assert float((own[0][4] - unit(down[:7]) * w["dkv.norm"]).abs().max()) < 1e-12
    assert float((own[1][4] - turned(down[7:], 4, 10.0, 4)).abs().max()) < 1e-12
    # the choice: negative scores, corrections that do not weigh, groups
    row = torch.tensor([[-0.9, -0.1, -0.3, -0.2, -0.8, -0.05]], dtype=torch.float64)
    none = torch.zeros(6, dtype=torch.float64)
    assert plain.choose(row, none, 2, None) == [[5, 1]]
    assert plain.choose(row, none, 2, dict(count=3, keep=1)) == [[5, 4]]
    assert plain.choose(row, none, 3, dict(count=3, keep=2)) == [[5, 1, 4]]
    assert plain.choose(row, torch.tensor([2.0, 0, 0, 0, 0, 0], dtype=torch.float64), 2, dict(count=2, keep=1)) == [[0, 1]]
    assert plain.choice_margin(row[0].tolist(), [5, 4], dict(count=3, keep=1)) == pytest.approx(0.05)
    assert plain.choice_margin(row[0].tolist(), [5, 1], None) == pytest.approx(0.1)
    # the mixture: an expert and an identity output, weights without renormalisation
    mlp = moe(3, 2, 5, identity=1)
    wm = {"router": rnd(4, W), "correction": torch.tensor([-9.0, -9.0, 0.0, 0.0], dtype=torch.float64)}
    for e in range(3):
        wm.update({f"e{e}.up": rnd(5, W), f"e{e}.down": rnd(W, 5)})
    out = plain.mixture(h, wm, mlp)
    for t in range(L):
        z = [math.exp(float(wm["router"][e] @ h[t])) for e in range(4)]
        up = [max(float(x), 0.0) ** 2 for x in wm["e2.up"] @ h[t]]
        want = z[2] / sum(z) * (wm["e2.down"] @ torch.tensor(up, dtype=torch.float64)) + z[3] / sum(z) * h[t]
        assert float((want - out[t]).abs().max()) < 1e-10


def test_a_random_folder_and_the_plain_model(tmp_path):
    helpers.make_folder(tmp_path, copy.deepcopy(RIKO_B), 7, store_dtype=torch.bfloat16)
    cfg, w = helpers.read_folder(str(tmp_path))
    assert w["l0.mix.pb"].shape == (6,) and w["l1.mlp.correction"].shape == (8,)
    assert float(w["l0.norm1"].float().abs().max()) < 0.6              # the distance from one
    streams = []
    logits = plain.forward(cfg, w, [3, 1, 4, 1, 5, 9, 2, 6], torch.float64, streams=streams)
    assert logits.shape == (8, 131) and bool(torch.isfinite(logits).all()) and len(streams) == 4


# ------------------------------------------------------------------ GPU
gpu = pytest.mark.gpu


def _sharpen(folder):
    """Rewrite a folder so that single keys weigh: the latent layers' scores are sharp (a softmax rests on one or two keys) and
    the sigmoid weights are nearly shut for most keys and open for a few."""
    from pulsar_b200.weights import safetensors_io
    cfg, w = helpers.read_folder(folder)
    for name in list(w):
        if name.endswith("mix.uq"):
            w[name] = (w[name].float() * 3.0).to(w[name].dtype)
        if name.endswith("mix.q.norm"):
            w[name] = (w[name].float() * 2.0).to(w[name].dtype)
        if name.endswith("mix.pb"):
            w[name] = (w[name].float() * 0.0 - 4.0).to(w[name].dtype)
    safetensors_io.write_safetensors(os.path.join(folder, "model.safetensors"), list(w.items()), metadata={"format": "pt"})


def _settle_routers(folder):
    """Rewrite a folder so that the corrections alone decide every router's choice (the same outputs for every token, another
    set in every layer): no rounding can change it, and the bfloat16 engine is held to the bar at every position."""
    from pulsar_b200.weights import safetensors_io
    cfg, w = helpers.read_folder(folder)
    gen = torch.Generator().manual_seed(1)
    for name in sorted(w):
        if name.endswith("mlp.correction"):
            w[name] = (2.0 * torch.randperm(w[name].numel(), generator=gen).float() - w[name].numel()).to(w[name].dtype)
    safetensors_io.write_safetensors(os.path.join(folder, "model.safetensors"), list(w.items()), metadata={"format": "pt"})


SHARP = config([
    layer(latent(3, 12, 6, 10, 28, 20)),
    layer(attention(4, 2, 16, 24, 8)),
    layer(latent(2, 8, 6, 16, 12, 20, kv_from=0)),
    layer(attention(2, 1, 8, 8, 8)),
], vocab=96, width=40)


SETTLED = ("A", "B", "C")


@pytest.fixture(scope="module")
def folders(tmp_path_factory):
    out = {}
    for name, raw in list(ALONE.items()) + [(n, c[0]) for n, c in CONFIGS.items()] + [("sharp", SHARP)] + [
            (f"{n} settled", CONFIGS[n][0]) for n in SETTLED]:
        d = tmp_path_factory.mktemp(f"riko{name}")
        # bfloat16 values: both precisions hold them exactly.  Wider weights than the default make every sublayer count.
        helpers.make_folder(d, copy.deepcopy(raw), 900 + len(out), store_dtype=torch.bfloat16, std=0.15)
        out[name] = str(d)
    _sharpen(out["sharp"])
    for n in SETTLED:
        _settle_routers(out[f"{n} settled"])
    return out


CLOSE_CALL = 0.05       # margin of a router's choice, relative to its largest score, below which bfloat16 rounding may choose otherwise


class _Reference(dict):
    """request -> plain logits; ``sure[request]``: the positions before the request's first close call of a router.  A token
    that is routed otherwise moves its own logits and, through its keys, those of the tokens behind it, so the bfloat16 engine
    is held to the bar up to there only (the float32 engine everywhere)."""
    sure = None


def _reference(folder, requests):
    cfg, w = helpers.read_folder(folder)
    ref = _Reference()
    ref.sure = {}
    for rid, toks in requests.items():
        margins = []
        ref[rid] = plain.forward(cfg, w, list(toks), torch.float64, log=margins)
        close = [int(torch.nonzero(m < CLOSE_CALL)[0]) for m in margins if bool((m < CLOSE_CALL).any())]
        ref.sure[rid] = min(close) if close else len(toks)
    return ref


def _replay(folder, dtype, trace, max_tokens, page_size, max_running=4):
    from pulsar_b200.replay import Replay
    rp = Replay(folder, dtype, max_tokens, page_size=page_size, max_running=max_running)
    got = {}
    for rec, rows in zip(trace.records, trace.rows):
        logits = rp.run_step(rec)
        for i, key in enumerate(rows):
            got[key] = logits[i]
    rp.cache.check_consistency()
    assert rp.cache.live_requests() == []
    assert all(f == g.allocator.n for f, g in zip(rp.cache.n_free_pages(), rp.cache.groups))
    return got, rp


def _compare(got, ref, dtype, what, tol=None):
    assert got
    worst = 0.0
    for (rid, pos), row in sorted(got.items()):
        if dtype == "bfloat16" and pos >= ref.sure[rid]:
            continue
        err = helpers.rel_err(row, ref[rid][pos])
        worst = max(worst, err)
        assert err < (tol or TOL[dtype]), f"{what}: request {rid} position {pos}: error {err:.3e} (first wrong place)"
    helpers.report(what, worst, dtype)


def _round64(n):
    return -(-n // 64) * 64


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(ALONE))
def test_each_mechanism_alone(folders, name, dtype):
    rng = random.Random(5)
    toks = helpers.random_tokens(rng, 45, 64)
    ref = _reference(folders[name], {"a": toks})
    for what, trace, page in (("whole", helpers.trace_whole(toks), 8), ("portions", helpers.trace_portions(toks, [5, 2, 11, 3, 2]), 4),
                              ("tail", helpers.trace_tail(toks, 20), 4)):
        got, _ = _replay(folders[name], dtype, trace, 64, page)
        _compare(got, ref, dtype, f"alone[{name}] {what}")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_prompt_tail_and_portions_agree_with_the_plain_logits(folders, name, dtype):
    raw, seed, page = CONFIGS[name]
    rng = random.Random(seed)
    toks = helpers.random_tokens(rng, 93, raw["vocab"])
    ref = _reference(folders[name], {"a": toks})
    for what, trace in (("whole", helpers.trace_whole(toks)), ("tail", helpers.trace_tail(toks, 60)),
                        ("portions", helpers.trace_portions(toks, [7, 2, 13, 2, 5, 17, 3])),
                        ("large portions", helpers.trace_portions(toks, [40, 18, 35])),
                        ("pairs", helpers.trace_portions(toks[:47], [2])), ("first tokens", helpers.trace_tail(toks[:12], 11))):
        got, _ = _replay(folders[name], dtype, trace, _round64(len(toks)), page)
        _compare(got, ref, dtype, f"{name} {what}")


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
@pytest.mark.parametrize("name", sorted(CONFIGS))
def test_mixed_batches_with_pages_and_slots_used_again(folders, name, dtype):
    raw, seed, page = CONFIGS[name]
    rng = random.Random(seed + 30)
    lengths = [40, 23, 64, 9, 31, 50, 17, 28, 45, 1, 2]
    requests = {f"r{i}": helpers.random_tokens(rng, n, raw["vocab"]) for i, n in enumerate(lengths)}
    ref = _reference(folders[name], requests)
    trace = helpers.trace_mixed(requests, rng, max_live=3)
    budget = sum(sorted(_round64(n) for n in lengths)[-3:])
    got, rp = _replay(folders[name], dtype, trace, budget, page, max_running=3)      # 11 requests through 3 slots
    assert len(got) == sum(lengths)
    _compare(got, ref, dtype, f"{name} mixed")


@gpu
@pytest.mark.parametrize("name", SETTLED)
def test_settled_routers_hold_the_bfloat16_engine_to_the_bar_everywhere(folders, name):
    raw, seed, page = CONFIGS[name]
    rng = random.Random(seed + 60)
    requests = {f"r{i}": helpers.random_tokens(rng, n, raw["vocab"]) for i, n in enumerate([150, 41, 9, 66, 20])}
    ref = _reference(folders[f"{name} settled"], requests)
    assert all(ref.sure[rid] == len(toks) for rid, toks in requests.items())
    long = requests["r0"]
    for what, trace, budget in (("whole", helpers.trace_whole(long, "r0"), 192), ("tail", helpers.trace_tail(long, 70, "r0"), 192),
                                ("portions", helpers.trace_portions(long, [2, 17, 33, 3, 5], "r0"), 192),
                                ("mixed", helpers.trace_mixed(requests, rng, max_live=3), 384)):
        got, _ = _replay(folders[f"{name} settled"], "bfloat16", trace, budget, page, max_running=3)
        _compare(got, ref, "bfloat16", f"{name} settled {what}")


@gpu
def test_a_batch_of_unequal_requests_equals_each_alone(folders):
    raw, seed, page = CONFIGS["A"]
    rng = random.Random(77)
    requests = {f"q{i}": helpers.random_tokens(rng, n, raw["vocab"]) for i, n in enumerate([37, 5, 22])}
    together = helpers.Trace()
    together.step([(rid, toks[:-4], range(len(toks) - 4)) for rid, toks in requests.items()])
    for k in range(4, 0, -1):
        together.step([(rid, toks[len(toks) - k:len(toks) - k + 1], [0]) for rid, toks in requests.items()],
                      end=list(requests) if k == 1 else [])
    both, _ = _replay(folders["A"], "float32", together, 3 * 64, page)
    for rid, toks in requests.items():
        alone, _ = _replay(folders["A"], "float32", helpers.trace_tail(toks, 4, rid), 64, page)
        for key, row in alone.items():
            assert helpers.rel_err(both[key], row) < 2e-6, f"{key}: a batch changed the logits"


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_long_decoding_and_a_long_prompt(folders, dtype):
    """230 tokens of which 220 are decoded one by one (from a captured graph), and 300 tokens at once (the bfloat16 engine's
    products for more than 128 rows)."""
    for name in ("A", "C", "D"):
        raw, seed, page = CONFIGS[name]
        rng = random.Random(9)
        toks = helpers.random_tokens(rng, 300, raw["vocab"])
        ref = _reference(folders[name], {"a": toks})
        got, rp = _replay(folders[name], dtype, helpers.trace_tail(toks[:230], 220), 256, page)
        _compare(got, ref, dtype, f"{name} long decoding")
        assert rp.runner.graph_replays > 150          # the steps of single tokens ran from a captured graph
        for what, trace in (("long prompt", helpers.trace_whole(toks)), ("long portions", helpers.trace_portions(toks, [140, 29, 131]))):
            got, _ = _replay(folders[name], dtype, trace, _round64(len(toks)), page)
            _compare(got, ref, dtype, f"{name} {what}")


def test_sharpened_weights_make_single_keys_count(monkeypatch):
    """The test below has teeth: with the sharpened weights a mask that loses one far key, values that are not turned back, a
    bias that is left out, or rows borrowed from nowhere move the plain logits by far more than the bar."""
    import tempfile
    with tempfile.TemporaryDirectory() as d:
        helpers.make_folder(d, copy.deepcopy(SHARP), 912, store_dtype=torch.bfloat16, std=0.15)
        _sharpen(d)
        cfg, w = helpers.read_folder(d)
    toks = helpers.random_tokens(random.Random(11), 120, 96)
    ref = plain.forward(cfg, w, toks, torch.float64)

    def moved(rows=slice(None)):
        return helpers.rel_err(plain.forward(cfg, w, toks, torch.float64)[rows], ref[rows])
    whole_mask, turn, rows_of = plain.causal, plain.rotate_neighbours, plain.latent_rows

    def lost_key(L):
        mask = whole_mask(L).clone()
        mask[100:, 7] = False
        return mask
    with monkeypatch.context() as mp:
        mp.setattr(plain, "causal", lost_key)
        assert moved(slice(100, None)) > 100 * TOL["float32"]
    with monkeypatch.context() as mp:
        mp.setattr(plain, "rotate_neighbours", lambda x, p, b, n, sign=1.0: x if sign < 0 else turn(x, p, b, n))
        assert moved() > 0.05
    with monkeypatch.context() as mp:
        mp.setattr(plain, "latent_rows", lambda *a: tuple(t.roll(1, 0) for t in rows_of(*a)))
        assert moved() > 0.05
    bias = {k: (v * 0 if k.endswith(".pb") else v) for k, v in w.items()}
    assert helpers.rel_err(plain.forward(cfg, bias, toks, torch.float64), ref) > 0.05


@gpu
@pytest.mark.parametrize("dtype", ["float32", "bfloat16"])
def test_sharp_scores_at_page_borders_and_far_back(folders, dtype):
    rng = random.Random(11)
    toks = helpers.random_tokens(rng, 330, 96)
    ref = _reference(folders["sharp"], {"a": toks})
    tol = TOL[dtype] * (2.0 if dtype == "bfloat16" else 1.5)       # sharp scores magnify the rounding of queries and keys
    for what, trace, page in (("whole", helpers.trace_whole(toks), 4), ("tail", helpers.trace_tail(toks, 40), 4),
                              ("portions", helpers.trace_portions(toks, [3, 2, 5, 9, 2, 31, 4]), 4),
                              ("tail, pages of 16", helpers.trace_tail(toks[:100], 70), 16)):
        got, _ = _replay(folders["sharp"], dtype, trace, _round64(len(toks)), page)
        _compare(got, ref, dtype, f"sharp {what}", tol)


def _step_context(q_lens, kv_lens):
    """What the kernels' wrappers read of a step: its device arrays, the lengths on the host, scratch memory."""
    cu = [0]
    for n in q_lens:
        cu.append(cu[-1] + n)
    i32 = lambda v: torch.tensor(v, dtype=torch.int32).cuda()
    return types.SimpleNamespace(cu_q=i32(cu), kv_len=i32(kv_lens), n_seqs=len(q_lens), n_tokens=cu[-1],
                                 host=types.SimpleNamespace(q_lens=list(q_lens)),
                                 seq_of_token=i32([s for s, n in enumerate(q_lens) for _ in range(n)]),
                                 scratch=lambda tag, shape, dtype=None: torch.empty(shape, dtype=dtype, device="cuda"))


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(6, 2, 64, 64), (4, 2, 128, 128), (2, 2, 64, 128), (3, 1, 192, 128), (4, 4, 12, 20), (5, 1, 40, 24), (2, 1, 7, 6)])
@pytest.mark.parametrize("lens", [([1, 1, 1], [1, 70, 301]), ([7, 1, 40], [7, 33, 200]), ([130], [130]), ([20, 33], [320, 33])])
def test_sigmoid_attention_against_its_formula(lens, sizes, dtype):
    """Every kernel of the general attention with sigmoid weights, a bias per head and rows that turn back.  Most scores are
    shut by the bias; for every query one key, often a far one, is made to stand out, so that losing it shows."""
    from pulsar_b200 import ops
    q_lens, kv_lens = lens
    H, G, D, V = sizes
    g = torch.Generator().manual_seed(sum(kv_lens) + D)
    rng = random.Random(D)
    n, page = sum(q_lens), 8
    pages = sum(-(-k // page) for k in kv_lens) + 3
    order = torch.randperm(pages, generator=g).tolist()
    k_pool, v_pool = torch.randn(pages, G, page, D, generator=g).to(dtype), torch.randn(pages, G, page, V, generator=g).to(dtype)
    tables, width = [], max(-(-k // page) for k in kv_lens)
    for k in kv_lens:
        m = -(-k // page)
        tables.append([order.pop() for _ in range(m)] + [-1] * (width - m))
    q = 0.3 * torch.randn(n, H, D, generator=g)
    bias = -4.0 + 0.5 * torch.randn(H, generator=g)
    ang = torch.rand(n, V // 2, generator=g) * 6.28
    cos, sin = torch.cos(ang), torch.sin(ang)
    scale, at = 1.0 / math.sqrt(D), 0
    rows = []
    for s, (ql, kl) in enumerate(zip(q_lens, kv_lens)):
        for i in range(ql):
            rows.append((at, s, kl - ql + i))
            at += 1
    for t, s, p in rows:                                             # one key stands out for every query and head
        j = rng.choice([0, 1, p, max(0, p - 1), rng.randrange(p + 1), (p // page) * page, max(0, (p // page) * page - 1)])
        for hd in range(H):
            key = k_pool[tables[s][j // page], hd // (H // G), j % page].float()
            q[t, hd] += 8.0 * math.sqrt(D) * key / (key * key).sum()
    want = torch.zeros(n, H, V, dtype=torch.float64)
    for t, s, p in rows:
        idx = torch.arange(p + 1)
        tb = torch.tensor(tables[s])
        for hd in range(H):
            kk = k_pool[tb[idx // page], hd // (H // G), idx % page].double()
            vv = v_pool[tb[idx // page], hd // (H // G), idx % page].double()
            o = torch.sigmoid(kk @ q[t, hd].double() * scale + float(bias[hd])) @ vv
            u, v = o[0::2].clone(), o[1::2].clone()
            o[0::2], o[1::2] = u * cos[t].double() + v * sin[t].double(), v * cos[t].double() - u * sin[t].double()
            want[t, hd] = o
    ctx = _step_context(q_lens, kv_lens)
    table = torch.tensor(tables, dtype=torch.int32).cuda()
    tc = dtype == torch.bfloat16 and (D, V) in ((64, 64), (64, 128), (128, 128), (192, 128))
    for form in [dict(tiled=False, tensor_cores=False), dict(tiled=True, tensor_cores=False)] + ([dict(tensor_cores=True)] if tc else []):
        for turn_back in (True, False):
            for out_dtype in {dtype, torch.float32}:
                out = torch.empty(n, H, V, dtype=out_dtype, device="cuda")
                ops.paged_attention_general(ctx, q.cuda(), k_pool.cuda(), v_pool.cuda(), out, table, scale, sigmoid=True, score_bias=bias.cuda(),
                                            turn_back=(cos.cuda(), sin.cuda()) if turn_back else None, **form)
                ref = want
                if not turn_back:                                    # the same rows, turned forward again
                    ref = want.clone()
                    c, s_ = cos.double()[:, None], sin.double()[:, None]
                    ref[..., 0::2], ref[..., 1::2] = want[..., 0::2] * c - want[..., 1::2] * s_, want[..., 1::2] * c + want[..., 0::2] * s_
                err = helpers.rel_err(out.float().cpu(), ref)
                assert err < (5e-3 if out_dtype == torch.bfloat16 else 2e-5), f"{form} turn_back={turn_back} {out_dtype}: {err:.3e}"


@gpu
def test_softmax_rows_turn_back_too():
    """The turning of the output does not depend on the kind of weights (all three kernels, and the splits' combination)."""
    from pulsar_b200 import ops
    g = torch.Generator().manual_seed(8)
    for q_lens, kv_lens in (([1, 1], [300, 40]), ([40], [90])):
        n, H, D, V, page = sum(q_lens), 2, 64, 64, 16
        ctx = _step_context(q_lens, kv_lens)
        width = -(-max(kv_lens) // page)
        table = torch.arange(len(q_lens) * width, dtype=torch.int32).view(len(q_lens), width).cuda()
        pool = torch.randn(2, len(q_lens) * width, 1, page, D, generator=g).to(torch.bfloat16).cuda()
        q, ang = torch.randn(n, H, D, generator=g).cuda(), torch.rand(n, V // 2, generator=g).cuda() * 6.28
        cos, sin = torch.cos(ang), torch.sin(ang)
        for form in (dict(tiled=False, tensor_cores=False), dict(tiled=True, tensor_cores=False), dict(tensor_cores=True)):
            flat, turned = torch.empty(n, H, V, device="cuda"), torch.empty(n, H, V, device="cuda")
            ops.paged_attention_general(ctx, q, pool[0], pool[1], flat, table, 0.125, **form)
            ops.paged_attention_general(ctx, q, pool[0], pool[1], turned, table, 0.125, turn_back=(cos, sin), **form)
            u, v = flat[..., 0::2], flat[..., 1::2]
            want = torch.empty_like(flat)
            want[..., 0::2], want[..., 1::2] = u * cos[:, None] + v * sin[:, None], v * cos[:, None] - u * sin[:, None]
            assert helpers.rel_err(turned.cpu(), want.cpu()) < 1e-6


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(4, 2, 12, 20, 8, True), (3, 3, 8, 6, 8, True), (2, 1, 7, 4, 6, True), (16, 4, 128, 128, 64, True),
                                   (5, 1, 16, 10, 6, False)])
def test_qk_prepare_whole_against_its_formula(sizes, dtype):
    from pulsar_b200 import ops
    H, G, D, V, rotary, neighbours = sizes
    g = torch.Generator().manual_seed(D)
    n, page, eps = 9, 4, 1e-5
    rows = torch.randn(n, (H + G) * D + G * V + 3, generator=g).to(dtype)
    qw, kw = torch.randn(H * D, generator=g), torch.randn(G * D, generator=g)
    ang, vang = torch.rand(n, rotary // 2, generator=g) * 6.28, torch.rand(n, V // 2, generator=g) * 6.28
    slots = torch.randperm(4 * page, generator=g)[:n].to(torch.int32)
    q_out = torch.empty(n, H, D, device="cuda")
    k_pool = torch.zeros(4, G, page, D, dtype=dtype, device="cuda")
    v_pool = torch.zeros(4, G, page, V, dtype=dtype, device="cuda")
    ops.qk_prepare_whole(rows.cuda(), q_out, k_pool, v_pool, slots.cuda(), H, G, D, V, page, qw.cuda(), kw.cuda(), eps,
                         (torch.cos(ang).cuda(), torch.sin(ang).cuda()), (torch.cos(vang).cuda(), torch.sin(vang).cuda()), neighbours)

    def turned(x, a, pairs):
        out, m = x.clone(), a.shape[1]
        c, s = torch.cos(a.double())[:, None], torch.sin(a.double())[:, None]
        lo, hi = (slice(0, 2 * m, 2), slice(1, 2 * m, 2)) if pairs else (slice(0, m), slice(m, 2 * m))
        out[..., lo], out[..., hi] = x[..., lo] * c - x[..., hi] * s, x[..., hi] * c + x[..., lo] * s
        return out
    r = rows.double()
    q = turned(plain.rms_norm(r[:, :H * D], qw.double(), eps).view(n, H, D), ang, neighbours)
    k = turned(plain.rms_norm(r[:, H * D:(H + G) * D], kw.double(), eps).view(n, G, D), ang, neighbours)
    v = turned(r[:, (H + G) * D:(H + G) * D + G * V].view(n, G, V), vang, neighbours)
    assert helpers.rel_err(q_out.cpu(), q) < 1e-6
    tol = 1e-6 if dtype == torch.float32 else 6e-3
    for t in range(n):
        p, o = int(slots[t]) // page, int(slots[t]) % page
        assert helpers.rel_err(k_pool[p, :, o].float().cpu(), k[t]) < tol
        assert helpers.rel_err(v_pool[p, :, o].float().cpu(), v[t]) < tol


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_latent_norms_against_their_formula(dtype):
    from pulsar_b200 import ops
    g = torch.Generator().manual_seed(6)
    tol = 1e-6 if dtype == torch.float32 else 6e-3
    n, q_rank, rank, rot, page = 10, 37, 21, 6, 4
    rows = torch.randn(n, q_rank + rank + rot + 2, generator=g).to(dtype)
    qw, kw, ang = torch.randn(q_rank, generator=g), torch.randn(rank, generator=g), torch.rand(n, rot // 2, generator=g) * 6.28
    slots = torch.randperm(3 * page, generator=g)[:n].to(torch.int32)
    pool = torch.zeros(3, 1, page, rank + rot, dtype=dtype, device="cuda")
    q_out, lat, rt = (torch.empty(n, w, dtype=dtype, device="cuda") for w in (q_rank, rank, rot))
    dev = rows.cuda()
    ops.latent_norms(dev[:, :q_rank], qw.cuda(), q_out, 1e-5, dev[:, q_rank:q_rank + rank + rot], kw.cuda(), torch.cos(ang).cuda(),
                     torch.sin(ang).cuda(), slots.cuda(), pool, rank, rot, page, lat, rt)
    r = rows.double()
    q_want, c_want = plain.rms_norm(r[:, :q_rank], qw.double(), 1e-5), plain.rms_norm(r[:, q_rank:q_rank + rank], kw.double(), 1e-5)
    tail = r[:, q_rank + rank:q_rank + rank + rot]
    u, v, c, s = tail[:, 0::2], tail[:, 1::2], torch.cos(ang.double()), torch.sin(ang.double())
    rot_want = torch.stack([u * c - v * s, v * c + u * s], dim=2).reshape(n, rot)
    assert helpers.rel_err(q_out.float().cpu(), q_want) < tol and helpers.rel_err(lat.float().cpu(), c_want) < tol
    assert helpers.rel_err(rt.float().cpu(), rot_want) < tol
    flat = pool.view(3 * page, rank + rot)
    assert torch.equal(flat[slots.cuda().long()], torch.cat([lat, rt], dim=1))
    free = [i for i in range(3 * page) if i not in slots.tolist()]
    assert float(flat[free].abs().max()) == 0.0
    again = torch.empty_like(q_out)
    ops.latent_norms(dev[:, :q_rank], qw.cuda(), again, 1e-5, None, None, torch.cos(ang).cuda(), torch.sin(ang).cuda(), None, None, rank, rot, page)
    assert torch.equal(again, q_out)


@gpu
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("sizes", [(1, 40, 6, 2, (3, 1)), (3, 48, 16, 4, (4, 2)), (40, 72, 12, 6, (2, 1)), (300, 64, 33, 1, (11, 3)),
                                   (20, 64, 8, 8, (4, 4)), (9, 32, 10, 3, None)])
def test_router_with_corrections_and_groups(sizes, dtype):
    from pulsar_b200 import ops
    n, W, E, top, groups = sizes
    g = torch.Generator().manual_seed(n + E)
    h = torch.randn(n, W, generator=g).to(dtype)
    router = torch.randn(E, W, generator=g)
    correction = 0.5 * torch.randn(E, generator=g) - 0.6             # most choice scores are negative
    ids = torch.empty(n, top, dtype=torch.int32, device="cuda")
    wts = torch.empty(n, top, device="cuda")
    ops.moe_route(h.cuda(), router.cuda(), ids, wts, softmax=True, correction=correction.cuda(), groups=groups)
    s = torch.softmax(h.double() @ router.double().T, dim=-1)
    chosen = plain.choose(s, correction.double(), top, None if groups is None else dict(count=groups[0], keep=groups[1]))
    assert ids.cpu().tolist() == chosen
    assert helpers.rel_err(wts.cpu(), torch.gather(s, 1, torch.tensor(chosen))) < 1e-5
    # the sigmoid router takes both, too
    ops.moe_route(h.cuda(), router.cuda(), ids, wts, 2.0, correction=correction.cuda(), groups=groups)
    s = torch.sigmoid(h.double() @ router.double().T)
    chosen = plain.choose(s, correction.double(), top, None if groups is None else dict(count=groups[0], keep=groups[1]))
    assert ids.cpu().tolist() == chosen
    assert helpers.rel_err(wts.cpu(), 2.0 * torch.gather(s, 1, torch.tensor(chosen))) < 1e-5


@gpu
@pytest.mark.parametrize("sizes", [(1, 40, 24, 3, 2, 2), (5, 64, 32, 4, 3, 1), (70, 72, 40, 5, 4, 3), (300, 128, 64, 6, 2, 2), (33, 64, 256, 2, 2, 0),
                                   (150, 256, 136, 3, 3, 4)])
def test_ungated_experts_against_their_formula(sizes):
    """The per-token kernels and both grouped forms; some tokens choose identity outputs only, one expert is chosen by nobody."""
    from pulsar_b200 import ops
    n, W, ff, E, top, identity = sizes
    g = torch.Generator().manual_seed(n)
    rng = random.Random(n)
    h = torch.randn(n, W, generator=g)
    up, down = torch.randn(E, ff, W, generator=g) / W ** 0.5, torch.randn(E, W, ff, generator=g) / ff ** 0.5
    usable = [e for e in range(E + identity) if e != 1 or E + identity <= top]
    ids = torch.tensor([rng.sample(usable, top) if t % 7 or identity < top else list(range(E, E + top)) for t in range(n)], dtype=torch.int32)
    wts = torch.rand(n, top, generator=g)
    for dtype in (torch.float32, torch.bfloat16):
        hd, ud, dd = h.to(dtype), up.to(dtype), down.to(dtype)
        want = torch.zeros(n, W, dtype=torch.float64)
        for t in range(n):
            for e, wt in zip(ids[t].tolist(), wts[t].tolist()):
                x = hd[t].double()
                want[t] += wt * (x if e >= E else dd[e].double() @ torch.relu(ud[e].double() @ x) ** 2)
        tol = 1e-5 if dtype == torch.float32 else 1e-2
        act = torch.empty(n * top, ff, dtype=dtype, device="cuda")
        out = torch.empty(n, W, dtype=dtype, device="cuda")
        ops.moe_up(hd.cuda(), ud.cuda(), ids.cuda(), act)
        ops.moe_down(act, dd.cuda(), ids.cuda(), wts.cuda(), None, out, identity=hd.cuda() if identity else None)
        assert helpers.rel_err(out.float().cpu(), want) < tol
        if dtype == torch.float32 or not ops.moe_grouped_supported(dtype, W, ff, E):
            continue
        for gathered in (None, torch.empty(n * top, W, dtype=dtype, device="cuda")):
            y = torch.empty(n * top, W, device="cuda")
            work = torch.empty(ops.moe_grouped_workspace(n, top, E), dtype=torch.int32, device="cuda")
            out.zero_()
            ops.moe_grouped(hd.cuda(), ud.cuda(), dd.cuda(), ids.cuda(), wts.cuda(), None, act, y, out, work, None, gathered, ungated=True,
                            identity=identity)
            assert helpers.rel_err(out.float().cpu(), want) < tol, f"gathered={gathered is not None}"
    ops.check_wait_words()


@gpu
@pytest.mark.parametrize("n,W,ff", [(1, 64, 48), (3, 96, 80), (8, 2048, 2048), (13, 128, 9728), (16, 80, 56), (40, 96, 72), (129, 64, 80),
                                    (300, 136, 520), (600, 256, 1024)])
def test_squared_relu_products(n, W, ff):
    from pulsar_b200 import ops
    g = torch.Generator().manual_seed(n)
    ctx = types.SimpleNamespace(scratch=lambda tag, shape, dtype=None: torch.empty(shape, dtype=dtype, device="cuda"))
    for dtype in (torch.float32, torch.bfloat16):
        h, w = torch.randn(n, W, generator=g).to(dtype), (torch.randn(ff, W, generator=g) / W ** 0.5).to(dtype)
        out = torch.empty(n, ff, dtype=dtype, device="cuda")
        ops.squared_relu_linear(ctx, h.cuda(), w.cuda(), out)
        want = torch.relu(h.double() @ w.double().T) ** 2
        assert helpers.rel_err(out.float().cpu(), want) < (1e-5 if dtype == torch.float32 else 5e-3)
        assert float(out.min()) >= 0.0
    ops.check_wait_words()


@gpu
def test_greedy_generation_through_the_engine(folders):
    from pulsar_b200.api import generate
    raw, seed, page = CONFIGS["A"]
    cfg, w = helpers.read_folder(folders["A"])
    rng = random.Random(41)
    prompts = [helpers.random_tokens(rng, n, raw["vocab"]) for n in (19, 4, 33)]

    def greedy(prompt, n_new):
        seq = list(prompt)
        for _ in range(n_new):
            seq.append(int(plain.forward(cfg, w, seq, torch.float64)[-1].argmax()))
        return seq[len(prompt):]
    got = generate(folders["A"], prompts, 12, dtype="float32", page_size=page, num_pages=40, max_sessions=4, max_running=2,
                   max_chunk_size=7, device="cuda:0")
    assert got == [greedy(p, 12) for p in prompts]
    # bfloat16 on the configuration without routers: every token lies within the bar of the plain model's best one
    raw, seed, page = CONFIGS["D"]
    cfg, w = helpers.read_folder(folders["D"])
    prompts = [helpers.random_tokens(rng, n, raw["vocab"]) for n in (19, 4, 33)]
    got16 = generate(folders["D"], prompts, 5, dtype="bfloat16", page_size=page, num_pages=40, max_sessions=4, max_running=3,
                     max_chunk_size=16, device="cuda:0")
    for p, new in zip(prompts, got16):
        seq = list(p)
        for tok in new:
            row = plain.forward(cfg, w, seq, torch.float64)[-1]
            assert float(row.max() - row[tok]) <= 2 * TOL["bfloat16"] * float(row.abs().max())
            seq.append(tok)


@gpu
def test_a_preempted_request_is_recomputed(folders):
    """More requests than pages: the scheduler preempts and recomputes; the tokens are those of undisturbed runs."""
    from pulsar_b200.api import generate
    raw, seed, page = CONFIGS["B"]
    rng = random.Random(43)
    prompts = [helpers.random_tokens(rng, n, raw["vocab"]) for n in (21, 30, 26, 17)]
    calm, tight = (generate(folders["B"], prompts, 20, dtype="float32", page_size=page, num_pages=pages, max_sessions=4, max_running=4,
                            max_chunk_size=16, device="cuda:0") for pages in (200, 36))
    assert tight == calm


@gpu
def test_command_line_and_trace_program(folders, tmp_path):
    """The framework's two programs on a Rikolix folder: greedy tokens from bin/pulsar-generate, and logits from
    bin/trace_run fed with steps on its standard input (a prompt in two portions, then single tokens)."""
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    raw, seed, page = CONFIGS["B"]
    cfg, w = helpers.read_folder(folders["B"])
    out = subprocess.run([sys.executable, os.path.join(root, "bin", "pulsar-generate"), "--model", folders["B"], "--dtype", "float32",
                          "--prompt_ids", "5,4,3,2,1,0,7", "--prompt_ids", "9 8", "--gen_tokens", "6", "--max_pages", "64", "--eos_id",
                          "-1", "--json"], capture_output=True, text=True, timeout=600)
    assert out.returncode == 0, out.stderr
    got = json.loads(out.stdout.strip().splitlines()[-1])["outputs"]
    for prompt, new in zip(([5, 4, 3, 2, 1, 0, 7], [9, 8]), got):
        seq = list(prompt)
        for tok in new:
            assert tok == int(plain.forward(cfg, w, seq, torch.float64)[-1].argmax())
            seq.append(tok)
    rng = random.Random(3)
    toks = helpers.random_tokens(rng, 40, raw["vocab"])
    trace = helpers.Trace()
    trace.step([("x", toks[:21], [20])])
    trace.step([("x", toks[21:37], [0, 15])])
    for i in range(37, 40):
        trace.step([("x", toks[i:i + 1], [0])], end=["x"] if i == 39 else [])
    run = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", folders["B"], "--dtype", "float32", "--out", str(tmp_path),
                          "--max-tokens", "64"], input=trace.lines(), capture_output=True, text=True, timeout=600)
    assert run.returncode == 0, run.stderr
    assert [ln for ln in run.stdout.splitlines() if ln.startswith("done ")] == [f"done {i}" for i in range(len(trace.records))]
    ref = plain.forward(cfg, w, toks, torch.float64)
    for i, rows in enumerate(trace.rows):
        got = torch.from_file(str(tmp_path / f"{i}.f32"), size=len(rows) * raw["vocab"], dtype=torch.float32).view(len(rows), -1)
        for j, (_, pos) in enumerate(rows):
            assert helpers.rel_err(got[j], ref[pos]) < TOL["float32"]
