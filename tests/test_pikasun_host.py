"""Host-side checks of the Pikasun configuration reader and of the host arithmetic beside its kernels: sizes and constants
come from the configuration alone, reused latents, the rotation's frequency rule, and how long portions are cut at chunks."""
import copy

import numpy as np
import pytest
import torch

import pikasun_plain as P
from mistralrs_b200 import engine, mixers, pikasun, registry


def latent(**kw):
    m = {"heads": 3, "dim": 4, "rot_dim": 6, "vdim": 5, "kv_rank": 7, "scale": 0.5, "rot": {"base": 100.0, "dims": 6}}
    m.update(kw)
    return {"type": "latent_attention", "mixer": m, "mlp": None}


def chunked(**kw):
    m = {"heads": 4, "kv_heads": 2, "dim": 8, "vdim": 6, "scale": 0.3, "mask": {"size": 5}, "rot": {"base": 100.0, "dims": 4}}
    m.update(kw)
    return {"type": "attention", "mixer": m, "mlp": {"kind": "dense", "ff": 9, "limit": 1.5}}


def cfg(layers, **kw):
    cj = {"architecture": "Pikasun", "vocab": 19, "width": 14, "norm": {"eps": 1e-4}, "logit_scale": 0.3, "logit_softcap": 4.0, "layers": layers}
    cj.update(kw)
    return cj


def test_shapes_follow_the_configuration():
    c = pikasun.PikasunConfig(cfg([chunked(), latent(), latent(kv_from=1, heads=2, vdim=9)]))
    s = c.tensor_shapes()
    assert (c.eps, c.logit_scale, c.logit_softcap) == (1e-4, 0.3, 4.0)
    assert s["embed"] == s["head"] == (19, 14) and s["final.norm"] == s["final.norm.b"] == (14,)
    assert s["l0.mix.q"] == (32, 14) and s["l0.mix.k"] == (16, 14) and s["l0.mix.v"] == (12, 14) and s["l0.mix.g"] == (4, 14)
    assert s["l0.mix.q.norm"] == s["l0.mix.q.b"] == (32,) and s["l0.mix.k.norm"] == s["l0.mix.k.b"] == (16,) and s["l0.mix.o"] == (14, 24)
    assert s["l1.mix.q"] == (30, 14) and s["l1.mix.dkv"] == (13, 14) and s["l1.mix.dkv.norm"] == (7,) and s["l1.mix.g"] == (15, 14)
    assert s["l2.mix.uk"] == (8, 7) and s["l2.mix.uv"] == (18, 7) and "l2.mix.dkv" not in s and "l2.mix.dkv.norm" not in s
    assert s["l0.norm2.b"] == (14,) and "l1.norm2" not in s and s["l0.mlp.gate"] == s["l0.mlp.up"] == (9, 14)
    assert set(pikasun.random_tensors(c, 1)) == set(s)


def test_what_does_not_fit_is_refused():
    for bad in ([latent(kv_from=0)], [chunked(), latent(kv_from=0)], [latent(), latent(kv_from=0), latent(kv_from=1)], [latent(), latent(kv_from=0, kv_rank=8)],
                [latent(), latent(kv_from=0, rot_dim=8)], [chunked(kv_heads=3)], [latent(rot={"base": 10.0, "dims": 8})]):
        with pytest.raises(ValueError):
            pikasun.PikasunConfig(cfg(bad))
    for key, val in (("type", "other"), ("mlp", {"kind": "moe"})):
        bad = latent()
        bad[key] = val
        with pytest.raises(NotImplementedError):
            pikasun.PikasunConfig(cfg([bad]))
    with pytest.raises(ValueError):
        pikasun.PikasunConfig(cfg([latent()], architecture="Other"))
    assert "Pikasun" in registry.registered()


def test_checkpoint_shapes_are_checked():
    c = pikasun.PikasunConfig(cfg([latent()]))
    t = pikasun.random_tensors(c, 1)
    for change in (lambda d: d.pop("l0.mix.uk"), lambda d: d.__setitem__("head", d["head"][:-1])):
        d = copy.copy(t)
        change(d)
        with pytest.raises((KeyError, ValueError)):
            pikasun.PikasunModel(c, d, torch.device("cpu"), torch.float32)


@pytest.mark.parametrize("dims,base,sc", [(16, 900.0, {"factor": 5.0, "original": 48, "fast": 3.0, "slow": 0.5}), (8, 10.0, {"factor": 1.0, "original": 4096, "fast": 32.0, "slow": 1.0}),
                                          (64, 1e6, {"factor": 40.0, "original": 300, "fast": 30.0, "slow": 2.0}), (2, 50.0, None), (12, 7.0, {"factor": 9.0, "original": 9, "fast": 1.5, "slow": 1.4})])
def test_rotation_frequencies(dims, base, sc):
    rot = {"dims": dims, "base": base}
    if sc:
        rot["scaling"] = sc
    f, mag = P.rotation_frequencies(rot)
    r = mixers.Rotation(dims, base, sc, torch.device("cpu"))
    assert torch.allclose(r.freq, f, rtol=1e-12) and abs(r.mag - mag) < 1e-12


def step(portions, page_size=4):
    """[(tokens, past)] -> StepBatch on the CPU."""
    tables, slot_map, first = [], [], 1
    for n, past in portions:
        pages = list(range(first, first + -(-(past + n) // page_size)))
        first += len(pages)
        tables.append(pages)
        slot_map += [pages[(past + i) // page_size] * page_size + (past + i) % page_size for i in range(n)]
    counts, pasts = [n for n, _ in portions], [p for _, p in portions]
    return engine.StepBatch(torch.device("cpu"), [0] * sum(counts), counts, pasts, list(range(len(counts))), tables, np.asarray(slot_map, dtype=np.int64), [])


@pytest.mark.parametrize("chunk", [0, 1, 7, 40, 64, 1000])
def test_dense_plan_covers_what_the_queries_see(chunk):
    """Every query row of a long portion is in exactly one segment, and its segment's keys up to it are the positions of its
    chunk; the gathered rows do not overlap; what is left out is listed."""
    portions = [(50, 0), (1, 12), (45, 33), (5, 3), (90, 128), (1, 0)]
    b = step(portions)
    plan = b.dense_plan(32, chunk)
    assert plan is b.dense_plan(32, chunk)                    # one per step
    segs, runs = plan.segments.view(-1, 4).tolist(), plan.runs.view(-1, 4).tolist()
    dense = {}
    for s, first, n, at in runs:
        for i in range(n):
            assert at + i not in dense
            dense[at + i] = (s, first + i)
    assert sorted(dense) == list(range(plan.n_rows))
    seen = {}
    for row, n, key0, before in segs:
        assert n <= plan.longest
        for i in range(n):
            assert row + i not in seen
            seen[row + i] = [dense[key0 + j] for j in range(before + i + 1)]
    at = 0
    for s, (n, past) in enumerate(portions):
        for i in range(n):
            lo = (past + i) // chunk * chunk if chunk else 0
            assert seen.pop(at + i, None) == ([(s, j) for j in range(lo, past + i + 1)] if n >= 32 else None)
        at += n
    assert not seen
    assert plan.rest_rows.tolist() == [50, 96, 97, 98, 99, 100, 191] and plan.rest == [(0, 1, 12, 1), (1, 5, 3, 3), (6, 1, 0, 5)]
    assert (plan.own_segments is None) == (chunk != 1)        # chunks of one position never reach back


def test_dense_plan_of_fresh_prompts_uses_the_steps_own_rows():
    b = step([(40, 0), (3, 9), (70, 0)])
    plan = b.dense_plan(32, 30)
    assert plan.own_segments.view(-1, 4).tolist() == [[0, 30, 0, 0], [30, 10, 30, 0], [43, 30, 43, 0], [73, 30, 73, 0], [103, 10, 103, 0]]
    aligned = step([(40, 60)])
    assert aligned.dense_plan(32, 30).own_segments is not None and aligned.dense_plan(32, 0).own_segments is None
    assert b.dense_plan(100, 0) is None
