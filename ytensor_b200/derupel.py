"""Host side of the Derupel language model: configuration and weights (padding, fusing) for the model handle of the C ABI
(ytcuda_derupel_*; native_lm.py has what it shares with other models).

The kernels want widths in multiples of 8, latents in multiples of 16 and, on the tensor cores, head dims of 64 or 128
(causal attention) and 128 (linear attention). Any other size is padded here with zero weights: padded channels of the
residual stream, of a head, a latent or a feed-forward stay zero, and norms run over the true widths."""
from __future__ import annotations

import ctypes as C
from dataclasses import dataclass, field

import numpy as np

from .native_lm import MLP_DENSE, MLP_MOE, MLP_NONE, NativeLM, up8, up_to

DECAYED, LATENT = 0, 1   # YTC_MIXER_*
MIXER_NAMES = {"lightning": DECAYED, "latent_attention": LATENT}


class _ConfigC(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("width", "norm_width", "vocab", "layers", "batch", "max_tokens", "chunk", "dtype")] + \
               [("eps", C.c_float), ("embed_scale", C.c_float)]


class _LayerC(C.Structure):
    _fields_ = [(n, C.c_int) for n in ("mixer", "heads", "dim", "vdim", "norm_width", "rot", "rot_dims", "head_ld", "rank",
                                       "q_rank", "q_width", "c_width", "mlp", "ff", "experts", "top", "shared_ff")] + \
               [(n, C.c_float) for n in ("scale", "limit", "shared_limit")]


@dataclass
class DerupelLayer:
    mixer: int
    heads: int
    dim: int                 # of a query / key head (the unrotated part, for latent attention)
    vdim: int
    decay: list = field(default_factory=list)  # linear attention: one per head
    rot_dim: int = 0         # latent attention
    rot_dims: int = 0        # rotated dimensions, the first of rot_dim
    rot_base: float = 10000.0
    kv_rank: int = 0
    q_rank: int = 0
    scale: float = 1.0
    mlp: int = MLP_NONE
    ff: int = 0              # dense width, or the width of one expert
    experts: int = 0
    top: int = 0
    limit: float = 0.0
    shared_ff: int = 0       # 0: no shared expert
    shared_limit: float = 0.0

    @staticmethod
    def from_dict(d: dict) -> "DerupelLayer":
        if d["type"] not in MIXER_NAMES:
            raise ValueError(f"unknown mixer '{d['type']}'")
        m = d["mixer"]
        L = DerupelLayer(mixer=MIXER_NAMES[d["type"]], heads=int(m["heads"]), dim=int(m["dim"]), vdim=int(m["vdim"]))
        if L.mixer == DECAYED:
            L.decay = [float(x) for x in m["decay"]]
            if len(L.decay) != L.heads:
                raise ValueError(f"{len(L.decay)} decays for {L.heads} heads")
        else:
            L.rot_dim, L.kv_rank, L.q_rank, L.scale = int(m["rot_dim"]), int(m["kv_rank"]), int(m["q_rank"]), float(m["scale"])
            L.rot_base, L.rot_dims = float(m["rot"]["base"]), int(m["rot"].get("dims", L.rot_dim))
            if L.rot_dims > L.rot_dim or L.rot_dims % 2:
                raise ValueError(f"{L.rot_dims} of {L.rot_dim} dimensions cannot be rotated")
        f = d.get("mlp")
        if f is None:
            return L
        if f["kind"] == "dense":
            L.mlp, L.ff = MLP_DENSE, int(f["ff"])
        elif f["kind"] == "moe":
            L.mlp, L.ff, L.limit = MLP_MOE, int(f["expert"]["ff"]), float(f["expert"]["limit"])
            L.experts, L.top = int(f["router"]["experts"]), int(f["router"]["top"])
            if f.get("shared"):
                L.shared_ff, L.shared_limit = int(f["shared"]["ff"]), float(f["shared"]["limit"])
        else:
            raise ValueError(f"unknown feed-forward '{f['kind']}'")
        return L

    def to_dict(self) -> dict:
        m = {"heads": self.heads, "dim": self.dim, "vdim": self.vdim}
        if self.mixer == DECAYED:
            m["decay"] = list(self.decay)
        else:
            m.update(rot_dim=self.rot_dim, kv_rank=self.kv_rank, q_rank=self.q_rank, scale=self.scale,
                     rot={"base": self.rot_base, "dims": self.rot_dims})
        f = None
        if self.mlp == MLP_DENSE:
            f = {"kind": "dense", "ff": self.ff}
        elif self.mlp == MLP_MOE:
            f = {"kind": "moe", "expert": {"ff": self.ff, "limit": self.limit},
                 "router": {"experts": self.experts, "top": self.top}}
            if self.shared_ff:
                f["shared"] = {"ff": self.shared_ff, "limit": self.shared_limit}
        return {"type": next(n for n, k in MIXER_NAMES.items() if k == self.mixer), "mixer": m, "mlp": f}


@dataclass
class DerupelConfig:
    width: int
    vocab: int
    eps: float
    embed_scale: float = 1.0
    layers: list = field(default_factory=list)

    @staticmethod
    def from_dict(d: dict) -> "DerupelConfig":
        return DerupelConfig(width=int(d["width"]), vocab=int(d["vocab"]), eps=float(d["norm"]["eps"]),
                             embed_scale=float(d["embedding"]["scale"]),
                             layers=[DerupelLayer.from_dict(x) for x in d["layers"]])

    def to_dict(self) -> dict:
        return {"architecture": "Derupel", "width": self.width, "vocab": self.vocab, "norm": {"eps": self.eps},
                "embedding": {"scale": self.embed_scale}, "layers": [x.to_dict() for x in self.layers]}

    def tensor_shapes(self) -> dict:
        """Checkpoint tensor names and shapes."""
        W, s = self.width, {"embed": (self.vocab, self.width)}
        for i, L in enumerate(self.layers):
            p, m = f"l{i}.", f"l{i}.mix."
            s[p + "norm1"] = (W,)
            hv = L.heads * L.vdim
            if L.mixer == DECAYED:
                s[m + "q"] = s[m + "k"] = (L.heads * L.dim, W)
                s[m + "v"] = (hv, W)
                s[m + "norm"] = (hv,)
            else:
                s[m + "dq"], s[m + "dq.norm"], s[m + "uq"] = (L.q_rank, W), (L.q_rank,), (L.heads * (L.dim + L.rot_dim), L.q_rank)
                s[m + "dkv"], s[m + "dkv.norm"] = (L.kv_rank + L.rot_dim, W), (L.kv_rank,)
                s[m + "uk"], s[m + "uv"] = (L.heads * L.dim, L.kv_rank), (hv, L.kv_rank)
            s[m + "g"], s[m + "o"] = (hv, W), (W, hv)
            if L.mlp == MLP_NONE:
                continue
            s[p + "norm2"] = (W,)
            if L.mlp == MLP_DENSE:
                s[p + "mlp.up"], s[p + "mlp.down"] = (L.ff, W), (W, L.ff)
                continue
            forms = [(f"e{e}", L.ff) for e in range(L.experts)] + ([("shared", L.shared_ff)] if L.shared_ff else [])
            for n, ff in forms:
                s[f"{p}mlp.{n}.gate"] = s[f"{p}mlp.{n}.up"] = (ff, W)
                s[f"{p}mlp.{n}.down"] = (W, ff)
            s[p + "mlp.router"] = (L.experts, W)
        s["final.norm"], s["head"] = (W,), (self.vocab, W)
        return s


@dataclass
class _Stored:
    """Sizes a layer is stored with."""
    dim: int
    vdim: int
    rot: int = 0
    head: int = 0
    rank: int = 0
    q_rank: int = 0


class DerupelForCausalLM(NativeLM):
    native = "derupel"

    def _stored(self, x: DerupelLayer) -> _Stored:
        bf16 = self.dtype == "bfloat16"
        if x.mixer == DECAYED:
            if bf16 and max(x.dim, x.vdim) <= 128:
                return _Stored(128, 128)
            return _Stored(up8(x.dim), up8(x.vdim))
        s = _Stored(up8(x.dim), up8(x.vdim), up_to(x.rot_dim, 16), 0, up_to(x.kv_rank, 16), up8(x.q_rank))
        s.head = s.dim + s.rot
        if bf16 and max(s.head, s.vdim) <= 128:
            s.head = s.vdim = 64 if max(s.head, s.vdim) <= 64 else 128
        return s

    def _create(self, chunk, dtype):
        cfg = self.cfg
        cc = _ConfigC(self.width_p, cfg.width, cfg.vocab, len(cfg.layers), self.batch, self.max_tokens, chunk, dtype, cfg.eps,
                      cfg.embed_scale)
        lc = (_LayerC * len(cfg.layers))()
        self.stored = [self._stored(x) for x in cfg.layers]
        for i, (x, s) in enumerate(zip(cfg.layers, self.stored)):
            lc[i] = _LayerC(x.mixer, x.heads, s.dim, s.vdim, x.heads * x.vdim, s.rot, x.rot_dims, s.head, s.rank, s.q_rank,
                            x.q_rank, x.kv_rank, x.mlp, up8(x.ff), x.experts, x.top, up8(x.shared_ff), x.scale, x.limit,
                            x.shared_limit)
        return cc, lc

    def _load(self, ck):
        cfg, wp, put = self.cfg, self.width_p, self._put
        for i, (x, s) in enumerate(zip(cfg.layers, self.stored)):
            p = f"l{i}."
            put("norm1", i, ck.vec(p + "norm1", wp))
            if x.mixer == DECAYED:
                self._load_decayed(ck, i, x, s)
            else:
                self._load_latent(ck, i, x, s)
            put("o", i, ck.heads_in(p + "mix.o", x.heads, x.vdim, s.vdim, wp))
            if x.mlp == MLP_NONE:
                continue
            put("norm2", i, ck.vec(p + "norm2", wp))
            fp = up8(x.ff)
            if x.mlp == MLP_DENSE:
                put("up", i, ck.mat(p + "mlp.up", fp, wp))
                put("down", i, ck.mat(p + "mlp.down", wp, fp))
                continue
            put("router", i, ck.mat(p + "mlp.router", cols=wp))
            up, down = ck.experts(p + "mlp.", x.experts, fp, wp)
            put("up", i, up)
            put("down", i, down)
            if x.shared_ff:
                sp = up8(x.shared_ff)
                put("shared_up", i, ck.gate_up(p + "mlp.shared.", sp, wp))
                put("shared_down", i, ck.mat(p + "mlp.shared.down", wp, sp))

    def _load_decayed(self, ck, i, x, s):
        torch, wp, p = self.torch, self.width_p, f"l{i}.mix."
        self._put("in", i, torch.cat([ck.heads_out(p + n, x.heads, d, dp, wp)
                                      for n, d, dp in (("q", x.dim, s.dim), ("k", x.dim, s.dim), ("v", x.vdim, s.vdim),
                                                       ("g", x.vdim, s.vdim))]))
        norm = ck.vec(p + "norm").reshape(x.heads, x.vdim)
        self._put("mix_norm", i, torch.nn.functional.pad(norm, (0, s.vdim - x.vdim)).reshape(-1))
        self._put("decay", i, torch.tensor(x.decay, dtype=torch.float32, device=ck.device))

    def _load_latent(self, ck, i, x, s):
        torch, wp, p = self.torch, self.width_p, f"l{i}.mix."
        pad = torch.nn.functional.pad
        dkv = ck.get(p + "dkv", torch.bfloat16)
        latent, key = dkv[:x.kv_rank], dkv[x.kv_rank:]
        rows = lambda a, n: pad(a, (0, wp - cfg_w, 0, n - a.shape[0]))  # noqa: E731
        cfg_w = self.cfg.width
        self._put("in", i, torch.cat([ck.mat(p + "dq", s.q_rank, wp), rows(latent, s.rank), rows(key, s.rot),
                                      ck.heads_out(p + "g", x.heads, x.vdim, s.vdim, wp)]))
        self._put("dq_norm", i, ck.vec(p + "dq.norm", s.q_rank))
        self._put("dkv_norm", i, ck.vec(p + "dkv.norm", s.rank))
        # a query head: dim unrotated dimensions, rot rotated ones, each part padded on its own
        uq = ck.get(p + "uq", torch.bfloat16).reshape(x.heads, x.dim + x.rot_dim, x.q_rank)
        head = torch.zeros(x.heads, s.head, s.q_rank, dtype=torch.bfloat16, device=ck.device)
        head[:, :x.dim, :x.q_rank] = uq[:, :x.dim]
        head[:, s.dim:s.dim + x.rot_dim, :x.q_rank] = uq[:, x.dim:]
        self._put("uq", i, head.reshape(x.heads * s.head, s.q_rank))
        uk = ck.heads_out(p + "uk", x.heads, x.dim, s.dim, s.rank)
        uv = ck.heads_out(p + "uv", x.heads, x.vdim, s.vdim, s.rank)
        self._put("uk", i, uk)
        self._put("uv", i, uv)
        # cache row [latent, rotated key part] -> every head's key and value in one product
        keys = torch.zeros(x.heads, s.head, s.rank + s.rot, dtype=torch.bfloat16, device=ck.device)
        keys[:, :s.dim, :s.rank] = uk.reshape(x.heads, s.dim, s.rank)
        keys[:, s.dim:s.dim + s.rot, s.rank:] = torch.eye(s.rot, dtype=torch.bfloat16, device=ck.device)
        self._put("expand", i, torch.cat([keys.reshape(x.heads * s.head, -1), pad(uv, (0, s.rot))]))
        n = x.rot_dims
        freq = np.power(float(x.rot_base), -2.0 * np.arange(max(1, n // 2)) / max(1, n)).astype(np.float32)
        self._put("freq", i, torch.from_numpy(freq).to(ck.device))
