"""Pikasun on the step engine against the plain float64 restatement (tests/pikasun_plain.py): every mechanism alone, then
whole prompts, token-by-token decoding, portions of many sizes, mixed batches, reused pages and slots, edges of the chunks, far
keys, long decoding, and greedy generation through the scheduler.  Small random configurations made here; f32 mode is held
to f32 rounding, bf16 mode to bf16 rounding."""
import copy
import json
import os
import subprocess
import sys

import numpy as np
import pytest
import torch

import pikasun_plain as P
from mistralrs_b200 import engine, mixers, pikasun, seq_ops as K

pytestmark = pytest.mark.gpu
F64 = torch.float64

YARN = {"factor": 5.0, "original": 48, "fast": 3.0, "slow": 0.5}


def dense(ff=52, limit=1.0):
    return {"kind": "dense", "ff": ff, "limit": limit}


def latent_layer(heads=4, dim=24, rot_dim=12, vdim=40, kv_rank=56, base=900.0, scaling=YARN, scale=0.2, rot_dims=None, kv_from=None, mlp=None):
    m = {"heads": heads, "dim": dim, "rot_dim": rot_dim, "vdim": vdim, "kv_rank": kv_rank, "scale": scale,
         "rot": {"base": base, "dims": rot_dims or rot_dim}}
    if scaling:
        m["rot"]["scaling"] = dict(scaling)
    if kv_from is not None:
        m["kv_from"] = kv_from
    return {"type": "latent_attention", "mixer": m, "mlp": mlp}


def chunk_layer(heads=6, kv_heads=2, dim=24, vdim=20, size=13, dims=10, base=300.0, scale=0.3, mlp=None):
    return {"type": "attention", "mixer": {"heads": heads, "kv_heads": kv_heads, "dim": dim, "vdim": vdim, "scale": scale, "mask": {"size": size},
                                           "rot": {"base": base, "dims": dims}}, "mlp": mlp}


def make_cfg(layers, width=72, vocab=131, eps=1e-5, logit_scale=0.7, cap=6.0):
    return {"architecture": "Pikasun", "vocab": vocab, "width": width, "norm": {"eps": eps}, "logit_scale": logit_scale, "logit_softcap": cap,
            "layers": layers}


FULL = make_cfg([chunk_layer(mlp=dense()), latent_layer(mlp=dense(limit=0.5)), latent_layer(kv_from=1, heads=2, dim=32, vdim=24, scale=0.15, mlp=None),
                 latent_layer(heads=3, dim=16, rot_dim=8, vdim=16, kv_rank=32, scaling=None, base=50.0, mlp=dense(ff=30)),
                 chunk_layer(heads=3, kv_heads=3, dim=16, vdim=32, size=50, dims=16, mlp=None),
                 latent_layer(kv_from=3, heads=5, dim=8, rot_dim=8, vdim=24, kv_rank=32, scaling=None, base=50.0, mlp=dense(limit=3.0)),
                 latent_layer(kv_from=1, heads=3, dim=16, vdim=16, mlp=dense())])
SMALL = make_cfg([latent_layer(mlp=None), chunk_layer(size=7, mlp=dense(ff=24)), latent_layer(kv_from=0, heads=1, mlp=dense())], logit_scale=1.0, cap=30.0)


def build(cj, dtype, device, seed=0, page_size=16, edit=None):
    cfg = pikasun.PikasunConfig(copy.deepcopy(cj))
    tensors = pikasun.random_tensors(cfg, seed)
    if edit:
        edit(tensors)
    model = pikasun.PikasunModel(cfg, tensors, device, dtype, page_size=page_size)
    return model, {k: v.to(F64) for k, v in tensors.items()}


def rel_err(got, want):
    """Per row: rms of the difference (mean taken off) over the rms of the wanted logits."""
    got, want = np.asarray(got, dtype=np.float64), np.asarray(want, dtype=np.float64)
    d = got - want
    d = d - d.mean(-1, keepdims=True)
    return np.sqrt((d ** 2).mean(-1)) / np.sqrt((want ** 2).mean())


TOL = {torch.float32: 1e-4, torch.bfloat16: 5e-2}


def assert_close(got, want, dtype, what=""):
    e = rel_err(got, want)
    assert e.max() < TOL[dtype], (what, float(e.max()), int(e.argmax()))


def replay(eng, prompts, schedule):
    """schedule: steps, each a list of (name, n_tokens).  Returns name -> logits of every position [T, vocab]."""
    live, rows = {}, {k: [] for k in prompts}
    for step in schedule:
        plan, want = [], []
        for name, n in step:
            if name not in live:
                live[name] = eng.new_request([])
            r = live[name]
            at = r.n_computed
            r.tokens.extend(prompts[name][at:at + n])
            plan.append((r, n))
            want.append(list(range(n)))
        lg = eng.execute(plan, want).cpu().numpy()
        at = 0
        for name, n in step:
            rows[name].append(lg[at:at + n])
            at += n
            if live[name].n_computed == len(prompts[name]):
                eng.finish(live.pop(name))
    return {k: np.concatenate(v) for k, v in rows.items() if v}


def tokens(n, vocab, seed):
    return np.random.default_rng(seed).integers(0, vocab, n).tolist()


def close_rows(got, want, tol):
    """Every row within tol; at bf16 tolerances 2 % of the rows may reach three times tol."""
    e = (got - want).norm(dim=-1) / want.norm(dim=-1).mean()
    if tol >= 1e-2:
        assert (e > tol).double().mean() <= 0.02 and e.max() < 3 * tol, (float(e.max()), int(e.argmax()))
    else:
        assert e.max() < tol, (float(e.max()), int(e.argmax()))


def seq_batch(device, portions, page_size=16):
    """One step of several sequences: portions = [(n_new, past, slot, first_page)]."""
    counts, pasts, slots, tables, slot_map = [], [], [], [], []
    for n, past, slot, first_page in portions:
        pages = list(range(first_page, first_page + -(-(past + n) // page_size)))
        counts.append(n), pasts.append(past), slots.append(slot), tables.append(pages)
        slot_map += [pages[(past + i) // page_size] * page_size + (past + i) % page_size for i in range(n)]
    return engine.StepBatch(device, [0] * sum(counts), counts, pasts, slots, tables, np.asarray(slot_map, dtype=np.int64), [])


def plain_mixer(layer, h, w, eps, p="l0.mix."):
    if layer["type"] == "attention":
        return P.chunked_attention(h, w, p, layer["mixer"], eps)
    return P.latent_attention(h, w, p, layer["mixer"], P.latent_rows(h, w, p, layer["mixer"], eps))


def run_mixer(cuda, mixer, h, portions, dtype, pages=80, page_size=16):
    """The mixer over `portions` of one sequence, on pages that held other data."""
    cache = mixer.alloc_cache(2, page_size * pages, dtype, cuda)
    for c in cache.values():
        c.normal_()
    got, at = [], 0
    for n in portions:
        got.append(mixer.forward(h[at:at + n].to(cuda).contiguous(), seq_batch(cuda, [(n, at, 1, 3)], page_size), cache).double().cpu())
        at += n
    return torch.cat(got)


def mixer_case(cuda, layer, dtype, portions, seed=3, edit=None, width=72, h=None):
    """Layer 0's mixer alone over `portions` of one sequence; returns (got [T, W], want [T, W])."""
    model, w = build(make_cfg([layer], width=width), dtype, cuda, seed, edit=edit)
    T = sum(portions)
    h = (torch.randn(T, width, generator=torch.Generator().manual_seed(seed)) if h is None else h).to(dtype)
    return run_mixer(cuda, model.layers[0].mixer, h, portions, dtype), plain_mixer(layer, h.double(), w, 1e-5)


# ---- mechanisms alone ------------------------------------------------------------------------------------------------
@pytest.mark.parametrize("width", [64, 45, 8, 1030])
@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_layer_norm_around_the_residual(cuda, width, dtype):
    """x += y, then the norm (mean taken off, bias added); inputs far from zero mean, so a mean left in or a variance around
    zero would show; and the norm of chosen rows only."""
    g = torch.Generator().manual_seed(width)
    T = 19
    x, y = torch.randn(T, width, generator=g) + 5.0, (torch.randn(T, width, generator=g) - 1.0).to(dtype)
    wt, b = torch.randn(width, generator=g), torch.randn(width, generator=g)
    norm = mixers.LayerNorm(wt.to(cuda), b.to(cuda), 1e-3)
    want = lambda v: P.layer_norm(v, wt.double(), b.double(), 1e-3)
    tol = 1e-5 if dtype == torch.float32 else 1e-2
    d = x.to(cuda)
    rows = torch.tensor([3, 3, 18, 0], dtype=torch.int32, device=cuda)
    close_rows(norm.of(d, dtype).double().cpu(), want(x.double()), tol)
    close_rows(norm.of(d, dtype, rows=rows).double().cpu(), want(x.double())[rows.long().cpu()], tol)
    h = norm.after_add(d, y.to(cuda)).double().cpu()
    new = x.double() + y.double()
    assert (d.double().cpu() - new).abs().max() < 1e-5
    close_rows(h, want(new), tol)


def test_layer_norm_of_nearly_equal_entries(cuda):
    """A large common offset over small differences: the squared deviations are taken around the mean, not as a difference of
    two large sums; and eps counts when the differences are tiny."""
    x = 100.0 + 0.01 * torch.randn(4, 96, generator=torch.Generator().manual_seed(1))
    one, zero = torch.ones(96, device=cuda), torch.zeros(96, device=cuda)
    for eps in (1e-10, 1e-3):
        got = mixers.LayerNorm(one, zero, eps).of(x.to(cuda), torch.float32).double().cpu()
        close_rows(got, P.layer_norm(x.double(), 1.0, 0.0, eps), 2e-2 if eps < 1e-9 else 1e-2)


def test_soft_cap(cuda):
    z = torch.linspace(-80.0, 80.0, 999)
    for dtype in (torch.float32, torch.bfloat16):
        for scale, cap in ((0.3, 7.0), (1.0, 100.0), (2.0, 0.5)):
            want = P.soft_cap(z.to(dtype).double() * scale, cap)
            assert (K.soft_cap(z.to(dtype).to(cuda), scale, cap).double().cpu() - want).abs().max() < 2e-6 * max(cap, 1.0)
    assert (K.soft_cap(z.to(cuda), 0.5, 0.0).cpu() - 0.5 * z).abs().max() < 1e-5        # no cap


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_feed_forward_caps_engage(cuda, dtype):
    """Large projections: the gate half is capped from above only, the other half on both sides, one is added to it."""
    def edit(t):
        for k in t:
            if k.endswith((".gate", ".up")):
                t[k].mul_(4.0)
    mlp = dense(ff=37, limit=0.75)
    model, w = build(make_cfg([latent_layer(mlp=mlp)]), dtype, cuda, 6, edit=edit)
    h = torch.randn(33, 72, generator=torch.Generator().manual_seed(6)).to(torch.bfloat16)
    want = P.capped_ff(h.double(), w, "l0.mlp.", 0.75)
    close_rows(model.layers[0].mlp.forward(h.to(dtype).to(cuda)).double().cpu(), want, 2e-5 if dtype == torch.float32 else 2e-2)
    assert (P.capped_ff(h.double(), w, "l0.mlp.", 1e9) - want).norm() > 0.2 * want.norm()


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 3e-2)])
@pytest.mark.parametrize("layer", [latent_layer(), chunk_layer()], ids=["latent", "chunked"])
@pytest.mark.parametrize("portions", [[150], [1] * 40, [7, 2, 33, 1, 64, 2, 41]])
def test_mixers_alone(cuda, layer, dtype, tol, portions):
    close_rows(*mixer_case(cuda, layer, dtype, portions), tol)


@pytest.mark.parametrize("layer", [latent_layer(heads=1, dim=8, rot_dim=2, vdim=8, kv_rank=8), latent_layer(heads=5, dim=7, rot_dim=6, vdim=9, kv_rank=11, scaling=None),
                                   latent_layer(heads=2, dim=64, rot_dim=32, vdim=64, kv_rank=160, rot_dims=14),
                                   latent_layer(heads=16, dim=16, rot_dim=8, vdim=136, kv_rank=264, scaling={"factor": 3.0, "original": 16, "fast": 2.0, "slow": 0.5}),
                                   chunk_layer(heads=1, kv_heads=1, dim=2, vdim=2, size=1, dims=2), chunk_layer(heads=4, kv_heads=4, dim=9, vdim=5, size=16, dims=4),
                                   chunk_layer(heads=4, kv_heads=1, dim=64, vdim=64, size=200, dims=64), chunk_layer(heads=2, kv_heads=1, dim=128, vdim=24, size=33, dims=6),
                                   chunk_layer(heads=6, kv_heads=3, dim=16, vdim=128, size=3, dims=8)])
@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 3e-2)])
def test_other_sizes(cuda, layer, dtype, tol):
    close_rows(*mixer_case(cuda, layer, dtype, [40, 1, 1, 3, 45], width=48), tol)


# (head size, value size, rotated size, rank): every combination of key boxes, shared part and value boxes the tcgen05 kernel is built for
TC_SIZES = [(64, 64, 8, 144), (32, 24, 24, 104), (48, 128, 16, 136), (128, 128, 64, 296), (96, 40, 32, 112), (112, 72, 8, 144), (16, 8, 40, 64), (64, 104, 64, 168)]


@pytest.mark.parametrize("dn,dv,dr,rank", TC_SIZES)
@pytest.mark.parametrize("portions", [[300], [70, 3, 130, 1, 1, 95]])
def test_latent_decompressed(cuda, dn, dv, dr, rank, portions, monkeypatch):
    """bf16 portions of 64 tokens or more decompress the latents they see and run on the tcgen05 kernel, whole prompts and later
    portions; the short ones between them stay in the absorbed form, on the same cache."""
    seen, real = [], K.tc_attention
    monkeypatch.setattr(K, "tc_attention", lambda *a, **k: (seen.append(1), real(*a, **k))[1])
    layer = latent_layer(heads=3, dim=dn, rot_dim=dr, vdim=dv, kv_rank=rank, scale=(dn + dr) ** -0.5)
    got, want = mixer_case(cuda, layer, torch.bfloat16, portions, width=64)
    assert len(seen) == sum(n >= 64 for n in portions)
    close_rows(got, want, 3e-2)
    assert K.tc_attention_timeouts() == 0


def test_latent_decompressed_beside_others(cuda):
    """One step: a prompt's start, a long portion that continues a second sequence, a short portion of a third and decoded
    tokens of two more; then the same with only fresh prompts and a decoded token."""
    layer = latent_layer(heads=5, dim=32, rot_dim=16, vdim=48, kv_rank=120)
    model, w = build(make_cfg([layer], width=64), torch.bfloat16, cuda, 7)
    mixer = model.layers[0].mixer
    cache = mixer.alloc_cache(5, 16 * 90, torch.bfloat16, cuda)
    cache["latent"].normal_()
    g = torch.Generator().manual_seed(7)
    hs = [torch.randn(n, 64, generator=g).to(torch.bfloat16) for n in (150, 230, 60, 12, 33)]
    first = [1, 12, 30, 40, 50]
    want = [plain_mixer(layer, h.double(), w, 1e-5) for h in hs]
    for step in ([(1, 0, 100), (2, 0, 41), (3, 0, 11), (4, 0, 31)], [(3, 11, 12), (1, 100, 230), (4, 31, 33), (0, 0, 66), (2, 41, 60)], [(0, 66, 67)], [(0, 67, 150)]):
        b = seq_batch(cuda, [(z - a, a, i, first[i]) for i, a, z in step])
        x = torch.cat([hs[i][a:z] for i, a, z in step]).to(cuda).contiguous()
        got = mixer.forward(x, b, cache).double().cpu()
        close_rows(got, torch.cat([want[i][a:z] for i, a, z in step]), 3e-2)


@pytest.mark.parametrize("layer", [chunk_layer(heads=4, kv_heads=2, dim=64, vdim=64, size=64, dims=20), chunk_layer(heads=3, kv_heads=1, dim=48, vdim=96, size=100, dims=48),
                                   chunk_layer(heads=2, kv_heads=2, dim=128, vdim=128, size=150, dims=64), chunk_layer(heads=5, kv_heads=1, dim=128, vdim=64, size=1000, dims=2),
                                   chunk_layer(heads=4, kv_heads=1, dim=64, vdim=64, size=40, dims=20), chunk_layer(heads=2, kv_heads=1, dim=128, vdim=128, size=9, dims=20)])
@pytest.mark.parametrize("portions", [[330], [90, 1, 70, 2, 167], [64, 64, 202], [33, 100, 32, 165]])
def test_chunked_long_portions(cuda, layer, portions):
    """bf16 portions of 32 tokens or more on tensor cores: chunks of 64 and more as segments of the tcgen05 kernel (portions that
    start at a chunk's border and inside one), smaller chunks of head sizes 64 / 128 masked in the mma.sync kernel."""
    close_rows(*mixer_case(cuda, layer, torch.bfloat16, portions, width=64), 3e-2)
    assert K.tc_attention_timeouts() == 0


def test_chunked_without_a_chunk_is_causal(cuda):
    layer = chunk_layer(heads=4, kv_heads=2, dim=64, vdim=64, dims=20)
    del layer["mixer"]["mask"]
    for dtype, tol in ((torch.float32, 3e-5), (torch.bfloat16, 3e-2)):
        close_rows(*mixer_case(cuda, layer, dtype, [90, 2, 1, 80]), tol)


@pytest.mark.parametrize("page_size", [4, 16, 64])
def test_chunked_several_sequences(cuda, page_size):
    layer = chunk_layer(heads=4, kv_heads=2, dim=32, vdim=48, size=70, dims=20)
    model, w = build(make_cfg([layer], width=64), torch.bfloat16, cuda, 7)
    mixer = model.layers[0].mixer
    mixer.page_size = page_size
    cache = mixer.alloc_cache(4, page_size * 300, torch.bfloat16, cuda)
    for c in cache.values():
        c.normal_()
    g = torch.Generator().manual_seed(7)
    hs = [torch.randn(n, 64, generator=g).to(torch.bfloat16) for n in (150, 230, 60, 12)]
    first = [1, 60, 130, 160]
    want = [plain_mixer(layer, h.double(), w, 1e-5) for h in hs]
    for step in ([(1, 0, 100), (2, 0, 41), (3, 0, 11)], [(3, 11, 12), (1, 100, 230), (0, 0, 66), (2, 41, 60)], [(0, 66, 150)]):
        b = seq_batch(cuda, [(z - a, a, i, first[i]) for i, a, z in step], page_size)
        got = mixer.forward(torch.cat([hs[i][a:z] for i, a, z in step]).to(cuda).contiguous(), b, cache).double().cpu()
        close_rows(got, torch.cat([want[i][a:z] for i, a, z in step]), 3e-2)


@pytest.mark.parametrize("rows", [1, 2, 7])
@pytest.mark.parametrize("heads,rank,dr", [(4, 64, 16), (20, 264, 24), (40, 520, 8)])
@pytest.mark.parametrize("context", [3, 64, 65, 700])
def test_latent_decode_shares_its_keys_among_ctas(cuda, rows, heads, rank, dr, context):
    """Small steps split a row tile's key tiles among CTAs and merge: the same numbers as one CTA, and as the plain softmax, for
    contexts below a tile, on its border and long; more shares than tiles."""
    g = torch.Generator().manual_seed(rank)
    ps, row = 16, -(-(rank + dr) // 8) * 8
    n_seq = 2
    tables = [list(range(1, 61)), list(range(61, 121))]
    latent = torch.randn(ps * 130, row, generator=g).to(torch.bfloat16).to(cuda)
    lens = [context + rows, max(1, context // 2) + rows]
    slot_map = [tables[s][(lens[s] - rows + i) // ps] * ps + (lens[s] - rows + i) % ps for s in range(n_seq) for i in range(rows)]
    b = engine.StepBatch(cuda, [0] * (n_seq * rows), [rows] * n_seq, [n - rows for n in lens], [0, 1], tables, np.asarray(slot_map, dtype=np.int64), [])
    qa = torch.randn(n_seq * rows, heads * (rank + dr), generator=g).to(torch.bfloat16).to(cuda)
    out = torch.full((n_seq * rows, heads * rank), float("nan"), dtype=torch.bfloat16, device=cuda)
    K.latent_prompt_attention(qa, latent, heads, rank, dr, 0.05, 0, b, ps, out)
    q = qa.double().cpu().view(n_seq, rows, heads, rank + dr)
    for s in range(n_seq):
        keys = torch.stack([latent[tables[s][j // ps] * ps + j % ps] for j in range(lens[s])]).double().cpu()
        for i in range(rows):
            vis = keys[:lens[s] - rows + i + 1]
            pr = torch.softmax(q[s, i] @ vis[:, :rank + dr].T * 0.05, dim=-1)
            want = pr @ vis[:, :rank]
            got = out.double().cpu().view(n_seq, rows, heads, rank)[s, i]
            assert (got - want).norm() < 1e-2 * want.norm()


def test_latent_cache_read_by_later_layers(cuda):
    """Mixers on one cache: the later ones have no latent projection of their own and see what the first stored, in prompts
    (decompressed or absorbed) and in decoding, through their own up-projections, scales and gates."""
    first, second = latent_layer(heads=3, dim=64, rot_dim=16, vdim=64, kv_rank=112), latent_layer(kv_from=0, heads=2, dim=32, rot_dim=16, vdim=48, kv_rank=112, scale=0.3)
    for dtype, tol in ((torch.float32, 3e-5), (torch.bfloat16, 3e-2)):
        model, w = build(make_cfg([first, second]), dtype, cuda, 5)
        assert "l1.mix.dkv" not in w and "l1.mix.uk" in w
        h = torch.randn(250, 72, generator=torch.Generator().manual_seed(5)).to(dtype)
        m0, m1 = model.layers[0].mixer, model.layers[1].mixer
        assert m1.alloc_cache(1, 16, dtype, cuda) == {}
        cache = m0.alloc_cache(1, 16 * 20, dtype, cuda)
        got = []
        for a, b in [(0, 100), (100, 101), (101, 102), (102, 120), (120, 250)]:
            batch = seq_batch(cuda, [(b - a, a, 0, 2)])
            m0.forward(h[a:b].to(cuda).contiguous(), batch, cache)
            got.append(m1.forward((2.0 * h[a:b]).to(cuda).contiguous(), batch, cache).double().cpu())    # its own input differs from the first one's
        rows = P.latent_rows(h.double(), w, "l0.mix.", first["mixer"], 1e-5)
        close_rows(torch.cat(got), P.latent_attention(2.0 * h.double(), w, "l1.mix.", second["mixer"], rows), tol)


# ---- keys made to stand out ---------------------------------------------------------------------------------------------
def pointed_chunk_edit(width, dim, heads, kv_heads):
    """Projections that copy the first `dim` inputs to every query and key and the NEXT entries to the values: a query scores
    high with exactly the keys whose input shares its direction there, and two tokens with one key still have two values."""
    def edit(t):
        eye = torch.eye(dim, width)
        t["l0.mix.q"].copy_(eye.repeat(heads, 1)), t["l0.mix.k"].copy_(eye.repeat(kv_heads, 1))
        dv = t["l0.mix.v"].shape[0] // kv_heads
        later = torch.zeros(dv, width)
        later[:dim, dim:2 * dim] = torch.eye(dim)[:dv]
        t["l0.mix.v"].copy_(later.repeat(kv_heads, 1))
        for n in ("q.b", "k.b"):
            t["l0.mix." + n].zero_()
        for n in ("q.norm", "k.norm"):
            t["l0.mix." + n].fill_(1.0)
    return edit


def pointed_latent_edit(width, dim, kv_rank, heads):
    """The latent copies the first kv_rank inputs, plain queries and keys its first `dim` entries, values the next ones; the
    rotated parts are zero."""
    def edit(t):
        dr = t["l0.mix.dkv"].shape[0] - kv_rank
        t["l0.mix.dkv"].copy_(torch.cat([torch.eye(kv_rank, width), torch.zeros(dr, width)]))
        t["l0.mix.q"].copy_(torch.cat([torch.eye(dim, width), torch.zeros(dr, width)]).repeat(heads, 1))
        t["l0.mix.uk"].copy_(torch.eye(dim, kv_rank).repeat(heads, 1))
        dv = t["l0.mix.uv"].shape[0] // heads
        later = torch.zeros(dv, kv_rank)
        later[:dim, dim:2 * dim] = torch.eye(dim)
        t["l0.mix.uv"].copy_(later.repeat(heads, 1))
        t["l0.mix.dkv.norm"].fill_(1.0)
    return edit


def pointed_inputs(T, width, dim, target, query, seed, longer=1.0):
    """Random inputs whose first `dim` entries are small except in `query` and `target`, which share a direction there (the
    target's `longer`) and differ elsewhere."""
    h = torch.randn(T, width, generator=torch.Generator().manual_seed(seed))
    h[:, :dim] *= 0.05
    h[query, :dim] = torch.randn(dim, generator=torch.Generator().manual_seed(seed + 1)) * 2.0
    h[target, :dim] = longer * h[query, :dim]
    return h


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("size", [64, 75, 20])
@pytest.mark.parametrize("inside", [True, False])
@pytest.mark.parametrize("how", ["prompt", "cut", "decoded"])
def test_chunk_edge_shows(cuda, dtype, size, inside, how):
    """A query near a chunk's end and one matching key: the chunk's first position (in sight) or the one before it (hidden).
    Chunks count from the sequence's start, however the prompt was cut."""
    dim = 16
    start = -(-150 // size) * size
    query, target = start + size - 3, start if inside else start - 1
    T = query + 1
    layer = chunk_layer(heads=2, kv_heads=1, dim=dim, vdim=16, size=size, scale=1.5)
    layer["mixer"]["rot"] = None
    h = pointed_inputs(T, 64, dim, target, query, 9)
    cuts = {"prompt": [T], "cut": [start - 7, 5, T - start + 2], "decoded": [start + 2, T - start - 5, 1, 1, 1]}[how]
    got, want = mixer_case(cuda, layer, dtype, cuts, width=64, h=h, edit=pointed_chunk_edit(64, dim, 2, 1))
    close_rows(got, want, 3e-5 if dtype == torch.float32 else 3e-2)
    _, w = build(make_cfg([layer], width=64), torch.float32, cuda, 3, edit=pointed_chunk_edit(64, dim, 2, 1))
    shifted = dict(layer["mixer"])
    first = P.chunk_start
    try:          # the plain model with the edge one position off
        P.chunk_start = lambda i, s: first(i, s) + (1 if inside else -1) if first(i, s) > 0 and i > first(i, s) else first(i, s)
        off = P.chunked_attention(h.to(dtype).double(), w, "l0.mix.", shifted, 1e-5)
    finally:
        P.chunk_start = first
    assert (off[-1] - want[-1]).norm() > 0.2 * want[-1].norm()


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
@pytest.mark.parametrize("target", [0, 15, 16, 17, 127, 128, 333])
@pytest.mark.parametrize("decoded", [False, True])
def test_far_key_among_hundreds(cuda, dtype, target, decoded):
    """One latent far back (the first token, both sides of a page's and of a key tile's border, somewhere in the middle) matches the last query."""
    T, dim, rank = 700, 16, 48
    layer = latent_layer(heads=2, dim=dim, rot_dim=8, vdim=24, kv_rank=rank, scale=1.0)
    edit = pointed_latent_edit(64, dim, rank, 2)
    h = pointed_inputs(T, 64, dim, target, T - 1, 13, longer=3.0)
    got, want = mixer_case(cuda, layer, dtype, [T - 2, 1, 1] if decoded else [T], width=64, h=h, edit=edit)
    close_rows(got[-3:], want[-3:], 3e-5 if dtype == torch.float32 else 3e-2)
    _, w = build(make_cfg([layer], width=64), torch.float32, cuda, 3, edit=edit)
    h[target] = torch.randn(64, generator=torch.Generator().manual_seed(1))
    assert (plain_mixer(layer, h.to(dtype).double(), w, 1e-5)[-1] - want[-1]).norm() > 0.2 * want[-1].norm()     # a lost key would show


@pytest.mark.parametrize("dtype,tol", [(torch.float32, 3e-5), (torch.bfloat16, 3e-2)])
def test_rotation_decides(cuda, dtype, tol):
    """The rotated parts alone decide the latent scores (the plain key part is zeroed); for the chunked layer all entries turn.
    Another pairing, or no magnitude on the scaled rotation, would show by far."""
    def edit(t):
        t["l0.mix.uk"].zero_()
    layer = latent_layer(heads=2, dim=16, rot_dim=16, vdim=16, kv_rank=40, scale=1.0, base=40.0)
    chunked = chunk_layer(heads=2, kv_heads=1, dim=16, vdim=16, size=90, dims=16, base=20.0, scale=0.6)
    for lay, ed in ((layer, edit), (chunked, None)):
        for portions in ([80], [17, 1, 1, 61]):
            got, want = mixer_case(cuda, lay, dtype, portions, edit=ed)
            close_rows(got, want, tol)
        _, w = build(make_cfg([lay]), torch.float32, cuda, 3, edit=ed)
        h = torch.randn(80, 72, generator=torch.Generator().manual_seed(3)).to(dtype).double()
        halves, neighbours, freq = P.rotate_halves, P.rotate_neighbours, P.rotation_frequencies
        try:
            P.rotate_halves, P.rotate_neighbours = neighbours, halves
            assert (plain_mixer(lay, h, w, 1e-5) - want).norm() > 0.1 * want.norm()
            P.rotate_halves, P.rotate_neighbours = halves, neighbours
            if lay is layer:
                P.rotation_frequencies = lambda rot: (freq(rot)[0], 1.0)
                assert (plain_mixer(lay, h, w, 1e-5) - want).norm() > 0.05 * want.norm()
        finally:
            P.rotate_halves, P.rotate_neighbours, P.rotation_frequencies = halves, neighbours, freq


def test_gates_and_whole_projection_norms_show(cuda):
    """Weights for which a gate left out, a gate of another head, or a norm per head instead of over the projection would show."""
    def spread(t):            # heads of very unequal size
        t["l0.mix.q"] *= torch.repeat_interleave(torch.tensor([0.2, 3.0, 1.0]), 16)[:, None].to(torch.bfloat16)
        t["l0.mix.q.b"] *= torch.repeat_interleave(torch.tensor([0.2, 3.0, 1.0]), 16).to(torch.bfloat16)
        t["l0.mix.g"] *= 3.0
    layer = chunk_layer(heads=3, kv_heads=3, dim=16, vdim=16, size=40, dims=8, scale=1.0)
    for portions in ([60], [31, 1, 28]):
        close_rows(*mixer_case(cuda, layer, torch.float32, portions, edit=spread), 3e-5)
    lat = latent_layer(heads=3, dim=16, vdim=16, kv_rank=64)
    for dtype, tol in ((torch.float32, 3e-5), (torch.bfloat16, 3e-2)):
        for portions in ([100], [70, 1, 29]):
            close_rows(*mixer_case(cuda, lat, dtype, portions, edit=lambda t: t["l0.mix.g"].mul_(3.0)), tol)


# ---- the model on the engine ----------------------------------------------------------------------------------------
@pytest.fixture(scope="module")
def full32(cuda):
    model, w = build(FULL, torch.float32, cuda, 11)
    prompts = {"a": tokens(150, 131, 1), "b": tokens(37, 131, 2), "c": tokens(2, 131, 3), "d": tokens(75, 131, 4), "e": tokens(1, 131, 5)}
    want = {k: P.forward(FULL, w, v).numpy() for k, v in prompts.items()}
    return model, prompts, want


def test_whole_prompts_and_layers(cuda, full32):
    model, prompts, want = full32
    eng = engine.Engine(model, max_tokens=160, max_seqs=1)
    for name in prompts:
        assert_close(replay(eng, prompts, [[(name, len(prompts[name]))]])[name], want[name], torch.float32, name)
    _, w = build(FULL, torch.float32, cuda, 11)
    layers, seen = [], []
    P.forward(FULL, w, prompts["b"], lambda i, x: layers.append(x.clone()))
    r = eng.new_request(prompts["b"])
    hooked = eng.execute([(r, 37)], after_layer=lambda i, x: seen.append(x.double().cpu())).cpu().numpy()
    eng.finish(r)
    assert len(seen) == len(layers) == 7
    for a, b in zip(seen, layers):
        assert (a - b).abs().max() < 1e-4 * b.abs().max()
    assert_close(hooked, want["b"][-1:], torch.float32)


def test_decode_token_by_token_equals_prefill(cuda, full32):
    model, prompts, want = full32
    eng = engine.Engine(model, max_tokens=160, max_seqs=1)
    assert_close(replay(eng, prompts, [[("b", 1)] for _ in range(37)])["b"], want["b"], torch.float32)
    got = replay(eng, prompts, [[("a", 40)]] + [[("a", 1)] for _ in range(110)])["a"]      # long decoding across chunks and pages
    assert_close(got, want["a"], torch.float32)


@pytest.mark.parametrize("sizes", [[2] * 75, [3, 16, 1, 15, 17, 2, 32, 31, 2, 2, 29], [149, 1], [16] * 9 + [6], [13] * 11 + [7], [50, 49, 51]])
def test_portions(cuda, full32, sizes):
    model, prompts, want = full32
    assert sum(sizes) == 150
    eng = engine.Engine(model, max_tokens=160, max_seqs=1)
    assert_close(replay(eng, prompts, [[("a", n)] for n in sizes])["a"], want["a"], torch.float32)


def test_mixed_batches_and_reuse(cuda, full32):
    """Unequal requests side by side, portions beside single tokens; the pools are too small for all of them at once, so
    pages and slots of finished requests are taken again (by requests that must not see what was left there)."""
    model, prompts, want = full32
    eng = engine.Engine(model, max_tokens=16 * 16, max_seqs=3)
    schedule = [[("a", 40), ("b", 30)], [("a", 1), ("b", 7), ("c", 2)], [("a", 60), ("d", 5)], [("d", 1), ("a", 1)], [("d", 69), ("a", 48), ("e", 1)]]
    got = replay(eng, prompts, schedule)
    for name in prompts:
        assert_close(got[name], want[name], torch.float32, name)
    assert eng.slots.num_free() == 3 and eng.pages.num_free_blocks() == 16
    again = replay(eng, prompts, [[("d", 75), ("b", 37), ("c", 2)], [("a", 100)], [("a", 50)]])    # every slot and page has been used before
    for name in ("a", "b", "d"):
        assert_close(again[name], want[name], torch.float32, name)


def test_a_request_may_sit_out_a_step(cuda, full32):
    model, prompts, want = full32
    eng = engine.Engine(model, max_tokens=16 * 16, max_seqs=2)
    got = replay(eng, prompts, [[("b", 20)], [("d", 30)], [("d", 1)], [("b", 2), ("d", 2)], [("d", 42)], [("b", 15)]])
    for name in ("b", "d"):
        assert_close(got[name], want[name], torch.float32, name)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_batch_of_decodes_matches_each_alone(cuda, dtype):
    """Also the captured-graph path: from its second occurrence a batch of single tokens replays a CUDA graph."""
    model, w = build(FULL, dtype, cuda, 11)
    prompts = {"a": tokens(150, 131, 1), "b": tokens(37, 131, 2), "d": tokens(75, 131, 4)}
    eng = engine.Engine(model, max_tokens=16 * 20, max_seqs=4)
    schedule = [[("a", 130), ("b", 17), ("d", 55)]] + [[("a", 1), ("b", 1), ("d", 1)] for _ in range(20)]
    got = replay(eng, prompts, schedule)
    for name in prompts:
        assert_close(got[name], P.forward(FULL, w, prompts[name]).numpy(), dtype, name)
    assert 3 in eng._graphs or not eng.decode_graphs


@pytest.mark.parametrize("page_size", [4, 64])
def test_other_page_sizes(cuda, page_size):
    model, w = build(SMALL, torch.float32, cuda, 21, page_size=page_size)
    p = {"x": tokens(90, 131, 8), "y": tokens(33, 131, 9)}
    eng = engine.Engine(model, max_tokens=192, max_seqs=2)
    got = replay(eng, p, [[("x", 50), ("y", 3)], [("x", 1), ("y", 30)], [("x", 39)]])
    for k in p:
        assert_close(got[k], P.forward(SMALL, w, p[k]).numpy(), torch.float32, k)


TENSOR_CORES = make_cfg([latent_layer(heads=3, dim=64, rot_dim=24, vdim=64, kv_rank=112, scale=0.1, mlp=dense()),
                         chunk_layer(heads=4, kv_heads=2, dim=64, vdim=64, size=90, dims=30, scale=0.125, mlp=dense(ff=96)),
                         latent_layer(kv_from=0, heads=2, dim=128, rot_dim=24, vdim=128, kv_rank=112, scale=0.08, mlp=None),
                         chunk_layer(heads=2, kv_heads=1, dim=128, vdim=128, size=30, dims=64, scale=0.09, mlp=dense())], width=128)


@pytest.mark.parametrize("cj", [FULL, TENSOR_CORES], ids=["small heads", "tensor-core heads"])
def test_bfloat16_model(cuda, cj):
    model, w = build(cj, torch.bfloat16, cuda, 11)
    p = {"a": tokens(320, 131, 1), "b": tokens(140, 131, 2), "c": tokens(70, 131, 3)}
    want = {k: P.forward(cj, w, v).numpy() for k, v in p.items()}
    schedules = ([[(k, len(p[k]))] for k in p], [[("a", 170), ("b", 5)], [("a", 1), ("b", 135)], [("a", 70), ("c", 70)], [("a", 79)]],
                 [[("a", 100), ("b", 100), ("c", 64)], [("c", 1), ("a", 199), ("b", 2)], [("c", 5), ("b", 1), ("a", 1)], [("b", 37), ("a", 20)]])
    for schedule in schedules:
        eng = engine.Engine(model, max_tokens=16 * 36, max_seqs=3)
        got = replay(eng, p, schedule)
        for k in got:
            assert_close(got[k], want[k][:len(got[k])], torch.bfloat16, k)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_one_layer_and_a_single_kind(cuda, dtype):
    """Models of one mixer kind only, without feed-forwards; constants that are neutral."""
    for layers in ([latent_layer()], [chunk_layer(size=5)], [chunk_layer(kv_heads=6, size=4096), chunk_layer(kv_heads=1)]):
        cj = make_cfg(layers, logit_scale=1.0, cap=1000.0)
        model, w = build(cj, dtype, cuda, 3)
        p = {"x": tokens(60, 131, 8)}
        got = replay(engine.Engine(model, max_tokens=64, max_seqs=1), p, [[("x", 40)], [("x", 1)], [("x", 19)]])
        assert_close(got["x"], P.forward(cj, w, p["x"]).numpy(), dtype)


AWKWARD = make_cfg([chunk_layer(heads=3, kv_heads=1, dim=9, vdim=5, size=11, dims=6, mlp=dense(ff=13)),
                    latent_layer(heads=3, dim=9, rot_dim=6, vdim=5, kv_rank=13, rot_dims=4, mlp=None),
                    latent_layer(kv_from=1, heads=1, dim=10, rot_dim=6, vdim=7, kv_rank=13, rot_dims=4, mlp=dense(ff=7))], width=45, vocab=77)


@pytest.mark.parametrize("dtype", [torch.float32, torch.bfloat16])
def test_sizes_that_align_with_nothing(cuda, dtype):
    """Odd width, head sizes, ranks and feed-forward sizes: every kernel falls back to its unvectorised path."""
    model, w = build(AWKWARD, dtype, cuda, 17)
    p = {"x": tokens(70, 77, 8), "y": tokens(33, 77, 9)}
    got = replay(engine.Engine(model, max_tokens=128, max_seqs=2), p, [[("x", 40), ("y", 3)], [("x", 1), ("y", 30)], [("x", 29)]])
    for k in p:
        assert_close(got[k], P.forward(AWKWARD, w, p[k]).numpy(), dtype, k)


def greedy_agrees(cj, w, prompt, out):
    """The plain model makes the same choices wherever its margin is clear."""
    seq = list(prompt)
    for t in out:
        lg = P.forward(cj, w, seq)[-1]
        top2 = lg.topk(2).values
        if top2[0] - top2[1] > 1e-3:
            assert int(lg.argmax()) == t
        seq.append(t)


def test_greedy_generation_through_the_scheduler(cuda):
    """engine.generate: waiting queue, admission by free slots and pages, chunked prefill under a small step budget,
    device top-1 sampling."""
    model, w = build(SMALL, torch.float32, cuda, 31)
    prompts = [tokens(n, 131, 40 + n) for n in (30, 5, 61, 1, 17)]
    eng = engine.Engine(model, max_tokens=16 * 8, max_seqs=2, max_step_tokens=24)
    outs = eng.generate(prompts, engine.SamplingParams(max_new_tokens=6))
    assert eng.slots.num_free() == 2 and eng.pages.num_free_blocks() == 8 and not eng.scheduler.running
    for p, out in zip(prompts, outs):
        assert len(out) == 6
        greedy_agrees(SMALL, w, p, out)


def test_model_folder_through_the_command_lines(cuda, tmp_path):
    """config.json + model.safetensors on disk -> the registry picks the class; the step-trace replay tool writes the
    logits it is asked for (requests cut into portions, a finished request's pages reused), and the generate command
    decodes greedily through the scheduler."""
    from safetensors.torch import save_file
    root = os.path.dirname(os.path.dirname(os.path.abspath(__file__)))
    cj = copy.deepcopy(SMALL)
    tensors = pikasun.random_tensors(pikasun.PikasunConfig(copy.deepcopy(cj)), 41)
    folder = tmp_path / "model"
    folder.mkdir()
    (folder / "config.json").write_text(json.dumps(cj))
    save_file({k: v.contiguous() for k, v in tensors.items()}, str(folder / "model.safetensors"))
    w = {k: v.to(F64) for k, v in tensors.items()}
    a, b = tokens(50, 131, 1), tokens(20, 131, 2)
    want_a, want_b = P.forward(cj, w, a).numpy(), P.forward(cj, w, b).numpy()
    steps = [{"step": 0, "entries": [{"id": "a", "tokens": a[:30], "want": [0, 29]}], "end": []},
             {"step": 1, "entries": [{"id": "a", "tokens": a[30:31], "want": []}, {"id": "b", "tokens": b[:19], "want": [18]}], "end": []},
             {"step": 2, "entries": [{"id": "b", "tokens": b[19:], "want": [0]}, {"id": "a", "tokens": a[31:], "want": [18]}], "end": ["a", "b"]},
             {"step": 3, "entries": [{"id": "c", "tokens": b, "want": [19]}], "end": ["c"]}]
    out = tmp_path / "out"
    r = subprocess.run([os.path.join(root, "bin", "trace_run"), "--model", str(folder), "--dtype", "float32", "--out", str(out), "--max-tokens", "128"],
                       input="\n".join(json.dumps(x) for x in steps) + "\n", capture_output=True, text=True, timeout=600)
    assert r.returncode == 0, r.stderr[-2000:]
    assert [x for x in r.stdout.split("\n") if x.startswith("done")] == ["done %d" % i for i in range(4)]
    read = lambda i: np.fromfile(out / ("%d.f32" % i), dtype="<f4").reshape(-1, 131)
    assert_close(read(0), want_a[[0, 29]], torch.float32)
    assert_close(read(1), want_b[[18]], torch.float32)
    assert_close(read(2), np.stack([want_b[19], want_a[49]]), torch.float32)
    assert_close(read(3), want_b[[19]], torch.float32)
    g = subprocess.run([sys.executable, os.path.join(root, "bin", "mrs-b200"), "generate", "--model", str(folder), "--dtype", "float32", "--max-new", "3",
                        "--prompt", " ".join(map(str, b))], capture_output=True, text=True, timeout=900)
    assert g.returncode == 0, g.stderr[-2000:]
    gen = json.loads(g.stdout.strip().split("\n")[-1])["generated"]
    assert len(gen) == 3
    greedy_agrees(cj, w, b, gen)
