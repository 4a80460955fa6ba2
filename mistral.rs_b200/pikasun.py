"""Pikasun: a decoder-only model with ONE f32 residual and layer norms (weight and bias) before every sublayer
(x <- x + sublayer(norm(x))), in which

  * the mixers are, in any order given by the configuration,
      `latent_attention`: keys and values of all heads decompressed from one RMS-normed latent per token, plus one rotated
                          key part the heads share (halves layout, YaRN-scaled frequencies); causal; a sigmoid gate per entry
                          of the concatenated heads; a later layer may reuse the cached latents (`kv_from`) with its own
                          up-projections;
      `attention`:        grouped-query attention with biased projections, query / key RMS norms over the whole projection,
                          rotary positions on part of each head in neighbouring pairs, chunks of `mask.size` positions that
                          see only themselves, a sigmoid gate per head;
  * the feed-forward is a gated one whose halves are capped, g * sigmoid(1.702 g) * (u + 1), or absent;
  * the logits have their own matrix, a multiplier and a soft cap.

Everything size-like comes from config.json: `vocab`, `width`, `norm.eps`, `logit_scale`, `logit_softcap` and per layer
`type`, `mixer` (its sizes and constants) and `mlp` (`kind` dense, or null).  Tensor names: `embed`, `l<i>.norm1|norm2`
(+ `.b`), `l<i>.mix.*`, `l<i>.mlp.*`, `final.norm` (+ `.b`), `head`.  The model is a composition of the mechanisms in
`mixers`; it has no cache or loop of its own — the engine owns pages and the step."""
import json
import os

import torch

from . import mixers as M
from . import seq_ops as K

ARCHITECTURE = "Pikasun"
MIXER_TYPES = ("latent_attention", "attention")
GATE_SLOPE, UP_SHIFT = 1.702, 1.0        # the feed-forward's joining rule: g * sigmoid(GATE_SLOPE * g) * (u + UP_SHIFT)


class PikasunConfig:
    def __init__(self, cj: dict):
        if cj.get("architecture") != ARCHITECTURE:
            raise ValueError(f"not a {ARCHITECTURE} configuration")
        self.raw = cj
        self.vocab, self.width = int(cj["vocab"]), int(cj["width"])
        self.eps = float(cj["norm"]["eps"])
        self.logit_scale = float(cj.get("logit_scale", 1.0))
        self.logit_softcap = float(cj.get("logit_softcap") or 0.0)
        self.layers = cj["layers"]
        for i, L in enumerate(self.layers):
            if L["type"] not in MIXER_TYPES:
                raise NotImplementedError(f"layer {i}: unknown mixer type {L['type']!r}")
            if L.get("mlp") is not None and L["mlp"]["kind"] != "dense":
                raise NotImplementedError(f"layer {i}: unknown feed-forward kind {L['mlp']['kind']!r}")
            m = L["mixer"]
            if L["type"] == "attention":
                if int(m["heads"]) % int(m.get("kv_heads", m["heads"])):
                    raise ValueError(f"layer {i}: heads must be a multiple of kv_heads")
                continue
            rot = m.get("rot")
            if rot and int(rot.get("dims", m["rot_dim"])) > int(m["rot_dim"]):
                raise ValueError(f"layer {i}: rot.dims exceeds rot_dim")
            if m.get("kv_from") is not None:
                src = int(m["kv_from"])
                S = self.layers[src] if 0 <= src < i else None
                if S is None or S["type"] != "latent_attention" or S["mixer"].get("kv_from") is not None:
                    raise ValueError(f"layer {i}: kv_from must name an earlier latent-attention layer that forms its own latent")
                for key in ("kv_rank", "rot_dim"):
                    if int(S["mixer"][key]) != int(m[key]):
                        raise ValueError(f"layer {i}: {key} differs from that of layer {src}, whose latent it reads")

    @classmethod
    def from_dir(cls, path):
        with open(os.path.join(path, "config.json")) as f:
            return cls(json.load(f))

    def tensor_shapes(self):
        """name -> shape of every checkpoint tensor (used to make random weights and to check a checkpoint)."""
        W, out = self.width, {}
        norm = lambda name: {name: (W,), name + ".b": (W,)}
        out["embed"], out["head"] = (self.vocab, W), (self.vocab, W)
        out.update(norm("final.norm"))
        for i, L in enumerate(self.layers):
            p, m = f"l{i}.", L["mixer"]
            out.update(norm(p + "norm1"))
            H, dk, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
            if L["type"] == "latent_attention":
                R, dr = int(m["kv_rank"]), int(m["rot_dim"])
                out.update({p + "mix.q": (H * (dk + dr), W), p + "mix.uk": (H * dk, R), p + "mix.uv": (H * dv, R), p + "mix.g": (H * dv, W),
                            p + "mix.o": (W, H * dv)})
                if m.get("kv_from") is None:
                    out.update({p + "mix.dkv": (R + dr, W), p + "mix.dkv.norm": (R,)})
            else:
                G = int(m.get("kv_heads", H))
                out.update({p + "mix.q": (H * dk, W), p + "mix.q.b": (H * dk,), p + "mix.k": (G * dk, W), p + "mix.k.b": (G * dk,),
                            p + "mix.v": (G * dv, W), p + "mix.v.b": (G * dv,), p + "mix.q.norm": (H * dk,), p + "mix.k.norm": (G * dk,),
                            p + "mix.g": (H, W), p + "mix.o": (W, H * dv)})
            mlp = L.get("mlp")
            if mlp is not None:
                ff = int(mlp["ff"])
                out.update(norm(p + "norm2"))
                out.update({p + "mlp.gate": (ff, W), p + "mlp.up": (ff, W), p + "mlp.down": (W, ff)})
        return out


class _Layer:
    pass


class PikasunModel:
    """Device-resident weights arranged for the kernels: projections that read the same input are one matrix (padded with
    zero rows so that its result's rows start on 16-byte boundaries), norm weights and biases are f32."""

    def __init__(self, cfg: PikasunConfig, tensors: dict, device, dtype=torch.bfloat16, page_size=16):
        if dtype not in K.DTYPE_CODE:
            raise ValueError("activation dtype must be bfloat16 or float32")
        self.cfg, self.device, self.dtype, self.page_size = cfg, device, dtype, page_size
        for name, shape in cfg.tensor_shapes().items():
            if name not in tensors:
                raise KeyError(f"checkpoint lacks tensor `{name}`")
            if tuple(tensors[name].shape) != tuple(shape):
                raise ValueError(f"tensor `{name}` has shape {tuple(tensors[name].shape)}, the configuration needs {tuple(shape)}")
        mat = lambda *names: torch.cat([tensors[n].to(device=device, dtype=dtype) for n in names], dim=0).contiguous()
        vec = lambda n: tensors[n].to(device=device, dtype=torch.float32).contiguous()
        norm = lambda n: M.LayerNorm(vec(n), vec(n + ".b"), cfg.eps)
        pad8 = lambda t: torch.cat([t, t.new_zeros(-t.shape[0] % 8, *t.shape[1:])]).contiguous()
        self.embed, self.head, self.final_norm = mat("embed"), mat("head"), norm("final.norm")
        self.layers, rotations = [], {}

        def rotation(rot, dims=None):
            if not rot:
                return None
            r = M.Rotation(rot.get("dims", dims), rot["base"], rot.get("scaling"), device)
            return rotations.setdefault(r.key, r)          # layers with equal constants share one table per step

        for i, L in enumerate(cfg.layers):
            p, m, lay = f"l{i}.", L["mixer"], _Layer()
            lay.norm1, lay.reads_cache_of = norm(p + "norm1"), None
            H, dk, dv = int(m["heads"]), int(m["dim"]), int(m["vdim"])
            if L["type"] == "latent_attention":
                shares = m.get("kv_from") is not None
                lay.reads_cache_of = int(m["kv_from"]) if shares else None
                parts = ("mix.q", "mix.g") if shares else ("mix.q", "mix.dkv", "mix.g")
                lay.mixer = M.LatentAttentionMixer(pad8(mat(*(p + n for n in parts))), None, mat(p + "mix.uk"), mat(p + "mix.uv"), mat(p + "mix.o"),
                                                   None, None if shares else vec(p + "mix.dkv.norm"), H, dk, int(m["rot_dim"]), dv, 0,
                                                   int(m["kv_rank"]), float(m["scale"]), 0, rotation(m.get("rot"), m["rot_dim"]), cfg.eps,
                                                   page_size, shares=shares, entry_gate=K.ACT_SIGMOID, pairing=K.PAIRS_HALVES)
            else:
                G, mask = int(m.get("kv_heads", H)), m.get("mask") or {}
                attn = M.WindowAttention(H, G, dk, dv, float(m["scale"]), 0, vec(p + "mix.q.norm"), vec(p + "mix.k.norm"), cfg.eps,
                                         norm_mode=K.QK_NORM_WHOLE, rotation=rotation(m.get("rot"), dk), page_size=page_size,
                                         chunk=int(mask.get("size", 0)), pairing=K.PAIRS_NEIGHBOURS)
                b_in = torch.cat([tensors[p + n].to(device=device, dtype=dtype) for n in ("mix.q.b", "mix.k.b", "mix.v.b")])
                lay.mixer = M.AttentionMixer(attn, pad8(mat(p + "mix.q", p + "mix.k", p + "mix.v", p + "mix.g")), mat(p + "mix.o"), page_size,
                                             b_in=pad8(torch.cat([b_in, b_in.new_zeros(H)])), gate_act=K.ACT_SIGMOID, gate_per_head=True)
            mlp, lay.mlp = L.get("mlp"), None
            if mlp is not None:
                lay.norm2 = norm(p + "norm2")
                lay.mlp = M.DenseGLU(mat(p + "mlp.gate", p + "mlp.up"), mat(p + "mlp.down"), K.GluRule.capped(float(mlp["limit"]), GATE_SLOPE, UP_SHIFT))
            self.layers.append(lay)

    # ---- loading ------------------------------------------------------------------------------------
    @classmethod
    def from_dir(cls, path, device, dtype=torch.bfloat16, page_size=16):
        from .nisasun import load_safetensors
        return cls(PikasunConfig.from_dir(path), load_safetensors(os.path.join(path, "model.safetensors")), device, dtype, page_size)

    @classmethod
    def random(cls, cfg: PikasunConfig, device, dtype=torch.bfloat16, seed=0, page_size=16):
        return cls(cfg, random_tensors(cfg, seed), device, dtype, page_size)

    # ---- the engine's interface ---------------------------------------------------------------------
    @property
    def vocab(self):
        return self.cfg.vocab

    def capturable(self, n_tok):
        """Every step launches a fixed sequence of kernels with no host read in between, so a decode step can be captured."""
        return True

    def alloc_caches(self, n_state_slots, n_token_slots):
        """Per layer: latent pages or key / value pages.  A layer that reuses another's latents holds a reference to that
        layer's pages."""
        caches = []
        for lay in self.layers:
            c = lay.mixer.alloc_cache(n_state_slots, n_token_slots, self.dtype, self.device)
            if lay.reads_cache_of is not None:
                c["latent"] = caches[lay.reads_cache_of]["latent"]
            caches.append(c)
        return caches

    def forward(self, batch, caches, after_layer=None):
        """Logits f32 [len(batch.rows), vocab] of one step's flat batch; advances `caches`.  after_layer(i, x) is called
        with the f32 residual after layer i (inspection only)."""
        T, W, n = batch.ids.numel(), self.cfg.width, len(self.layers)
        x = K.embed_scaled(self.embed, batch.ids, 1.0, torch.empty(T, W, dtype=torch.float32, device=self.device))
        h = self.layers[0].norm1.of(x, self.dtype)
        for i, lay in enumerate(self.layers):
            y = lay.mixer.forward(h, batch, caches[i])
            if lay.mlp is not None:
                y = lay.mlp.forward(lay.norm2.after_add(x, y))
            if i + 1 < n:
                h = self.layers[i + 1].norm1.after_add(x, y)
            else:
                K.rms_residual(x, y, dst=x)
            if after_layer is not None:
                after_layer(i, x)
        hn = self.final_norm.of(x, self.dtype, rows=batch.rows)
        return K.soft_cap(M.linear(hn, self.head), self.cfg.logit_scale, self.cfg.logit_softcap)


def random_tensors(cfg: PikasunConfig, seed=0):
    """Random bf16-representable weights with activations of order one (throughput runs and tests)."""
    g = torch.Generator().manual_seed(seed)
    out = {}
    for name, shape in cfg.tensor_shapes().items():
        leaf = name.split(".")[-1]
        if leaf in ("norm1", "norm2", "norm"):
            t = 1.0 + 0.1 * torch.randn(shape, generator=g)
        elif leaf == "b":
            t = 0.2 * torch.randn(shape, generator=g)
        elif name == "embed":
            t = torch.randn(shape, generator=g)
        else:
            t = torch.randn(shape, generator=g) / shape[-1] ** 0.5
        out[name] = t.to(torch.bfloat16)
    return out
