"""Configuration of the Milivik decoder: every size and constant comes from ``config.json``."""
from __future__ import annotations

from dataclasses import dataclass, field

import torch

from ...ops.latent_attention import LatentShape
from ...ops.lm import HeadShape, QueryGrowth
from ...ops.moe import Router
from ...ops.stream import Yarn
from ..packed_decoder import round_up
from ..seq_table import StateTensor


@dataclass
class LatentMixer:
    """Latent attention with a latent on the query side, a sliding window and a gate on every output channel."""
    shape: LatentShape
    q_rank: int
    scale: float
    rot_base: float
    yarn: Yarn | None
    window: int | None              # None = every earlier position

    @classmethod
    def from_dict(cls, d: dict) -> "LatentMixer":
        rot, mask = d["rot"], d.get("mask") or {}
        sc = rot.get("scaling")
        yarn = None if sc is None else Yarn(float(sc["factor"]), float(sc["original"]), float(sc["fast"]), float(sc["slow"]))
        m = cls(LatentShape(int(d["heads"]), int(d["dim"]), int(d["rot_dim"]), int(d["vdim"]), int(d["kv_rank"])),
                int(d["q_rank"]), float(d["scale"]), float(rot["base"]), yarn,
                None if mask.get("size") is None else int(mask["size"]))
        if m.shape.rot % 2:
            raise ValueError(f"rot_dim must be even, got {m.shape.rot}")
        if int(rot.get("dims", m.shape.rot)) != m.shape.rot:
            raise ValueError(f"rot.dims ({rot['dims']}) must equal rot_dim ({m.shape.rot})")
        if m.window is not None and m.window < 1:
            raise ValueError(f"mask.size must be positive, got {m.window}")
        return m

    @property
    def q_rank_p(self) -> int:
        return round_up(self.q_rank, 16)


@dataclass
class DiffMixer:
    """Differential attention: two maps per head over the same values."""
    heads: int
    kv_heads: int
    dim: int
    vdim: int
    scale: float
    diff: float
    growth: QueryGrowth | None

    @classmethod
    def from_dict(cls, d: dict) -> "DiffMixer":
        t = d.get("q_temp")
        m = cls(int(d["heads"]), int(d["kv_heads"]), int(d["dim"]), int(d["vdim"]), float(d["scale"]), float(d["diff"]),
                None if t is None else QueryGrowth(float(t["coef"]), float(t["every"])))
        if m.heads % m.kv_heads:
            raise ValueError(f"heads ({m.heads}) must be a multiple of kv_heads ({m.kv_heads})")
        if m.growth is not None and m.growth.every <= 0:
            raise ValueError(f"q_temp.every must be positive, got {m.growth.every}")
        return m

    @property
    def head_shape(self) -> HeadShape:
        """Every map is a head of its own on the query and key side."""
        return HeadShape(2 * self.heads, 2 * self.kv_heads, self.dim, self.vdim, round_up(self.dim, 16), round_up(self.vdim, 16),
                         v_heads=self.kv_heads)


@dataclass
class DenseConfig:
    ff: int


@dataclass
class ExpertsConfig:
    router: Router
    ff: int
    shared_ff: int | None = None    # None = no shared expert

    @classmethod
    def from_dict(cls, d: dict) -> "ExpertsConfig":
        r = d["router"]
        g = r.get("groups") or {}
        router = Router(int(r["experts"]), int(r["top"]), True, int(g.get("count", 0)), int(g.get("keep", 0)), float(r.get("scale", 1.0)))
        return cls(router, int(d["expert"]["ff"]), int(d["shared"]["ff"]) if d.get("shared") else None)


def _feed_forward(d: dict | None) -> DenseConfig | ExpertsConfig | None:
    if d is None:
        return None
    if d.get("kind") == "dense":
        return DenseConfig(int(d["ff"]))
    if d.get("kind") == "moe":
        return ExpertsConfig.from_dict(d)
    raise ValueError(f"unknown feed-forward kind {d.get('kind')!r}")


@dataclass
class LayerConfig:
    mixer: LatentMixer | DiffMixer
    mlp: DenseConfig | ExpertsConfig | None = None


_MIXERS = {"latent_attention": LatentMixer, "attention": DiffMixer}


@dataclass
class MilivikConfig:
    vocab_size: int
    hidden_size: int
    norm_eps: float
    embed_scale: float
    logit_scale: float
    layers: list[LayerConfig] = field(default_factory=list)

    # what the engine reads from any decoder configuration
    mrope_section = None

    @classmethod
    def from_dict(cls, d: dict) -> "MilivikConfig":
        layers = []
        for i, e in enumerate(d["layers"]):
            if e["type"] not in _MIXERS:
                raise ValueError(f"layer {i}: unknown mixer type {e['type']!r}")
            try:
                layers.append(LayerConfig(_MIXERS[e["type"]].from_dict(e["mixer"]), _feed_forward(e.get("mlp"))))
            except ValueError as err:
                raise ValueError(f"layer {i}: {err}") from None
        return cls(int(d["vocab"]), int(d["width"]), float(d["norm"]["eps"]), float(d["embedding"]["scale"]), float(d["logit_scale"]),
                   layers)

    @property
    def num_hidden_layers(self) -> int:
        return len(self.layers)

    @property
    def padded_width(self) -> int:
        return round_up(self.hidden_size, 8)

    def _mlp_max(self, kind, f) -> int:
        return max((f(l.mlp) for l in self.layers if isinstance(l.mlp, kind)), default=0)

    @property
    def num_experts(self) -> int:
        return self._mlp_max(ExpertsConfig, lambda m: m.router.experts)

    @property
    def num_experts_per_tok(self) -> int:
        return self._mlp_max(ExpertsConfig, lambda m: m.router.top)

    @property
    def moe_intermediate_size(self) -> int:
        return self._mlp_max(ExpertsConfig, lambda m: m.ff)

    @property
    def intermediate_size(self) -> int:
        return max(self._mlp_max(DenseConfig, lambda m: m.ff), self._mlp_max(ExpertsConfig, lambda m: m.shared_ff or 0))

    def kv_layer_shapes(self) -> list[tuple[int, int, int]]:
        """(heads, key channels, value channels) of every layer's pages: one row of latent and rotated key part, whose first
        channels are also the value; or per KV head the keys of both maps side by side and one value."""
        out = []
        for l in self.layers:
            if isinstance(l.mixer, LatentMixer):
                out.append((1, l.mixer.shape.row, 0))
            else:
                hs = l.mixer.head_shape
                out.append((hs.values, 2 * hs.dp, hs.vp))
        return out

    def state_shapes(self) -> list[tuple[StateTensor, ...]]:
        return [() for _ in self.layers]

    def tensor_shapes(self) -> dict[str, tuple[int, ...]]:
        """Checkpoint tensor names and shapes."""
        D = self.hidden_size
        t: dict[str, tuple[int, ...]] = {"embed": (self.vocab_size, D), "final.norm": (D,)}

        def gated(p, ff):
            t[p + "gate"], t[p + "up"], t[p + "down"] = (ff, D), (ff, D), (D, ff)
        for i, l in enumerate(self.layers):
            p, m = f"l{i}.", l.mixer
            t[p + "norm1"] = (D,)
            if isinstance(m, LatentMixer):
                s = m.shape
                t[p + "mix.dq"], t[p + "mix.dq.norm"] = (m.q_rank, D), (m.q_rank,)
                t[p + "mix.uq"] = (s.heads * (s.dim + s.rot), m.q_rank)
                t[p + "mix.dkv"], t[p + "mix.dkv.norm"] = (s.rank + s.rot, D), (s.rank,)
                t[p + "mix.uk"], t[p + "mix.uv"] = (s.heads * s.dim, s.rank), (s.heads * s.vdim, s.rank)
                t[p + "mix.g"], t[p + "mix.o"] = (s.heads * s.vdim, D), (D, s.heads * s.vdim)
            else:
                t[p + "mix.q"], t[p + "mix.k"] = (m.heads * 2 * m.dim, D), (m.kv_heads * 2 * m.dim, D)
                t[p + "mix.v"] = (m.kv_heads * m.vdim, D)
                for n in ("q.norm", "k.norm", "lq1", "lk1", "lq2", "lk2"):
                    t[p + "mix." + n] = (m.dim,)
                t[p + "mix.g"], t[p + "mix.o"] = (m.heads, D), (D, m.heads * m.vdim)
            if l.mlp is not None:
                t[p + "norm2"] = (D,)
            if isinstance(l.mlp, DenseConfig):
                gated(p + "mlp.", l.mlp.ff)
            elif l.mlp is not None:
                t[p + "mlp.router"] = (l.mlp.router.experts, D)
                for e in range(l.mlp.router.experts):
                    gated(f"{p}mlp.e{e}.", l.mlp.ff)
                if l.mlp.shared_ff:
                    gated(p + "mlp.shared.", l.mlp.shared_ff)
                    t[p + "mlp.shared.sg"] = (1, D)
        return t


def tiny_config_dict(**over) -> dict:
    """A small geometry for tests and smoke runs; no two sizes are equal."""
    moe = {"kind": "moe", "expert": {"ff": 56}, "shared": {"ff": 88},
           "router": {"experts": 12, "top": 4, "scale": 1.7, "groups": {"count": 3, "keep": 2}}}
    latent = {"heads": 3, "dim": 24, "rot_dim": 12, "vdim": 40, "kv_rank": 48, "q_rank": 64, "scale": 0.17, "mask": {"size": 21},
              "rot": {"base": 7000.0, "dims": 12, "scaling": {"factor": 3.0, "original": 256, "fast": 16.0, "slow": 2.0}}}
    diff = {"heads": 6, "kv_heads": 2, "dim": 20, "vdim": 36, "scale": 0.2, "diff": 0.35, "q_temp": {"coef": 0.2, "every": 15}}
    d = {"architecture": "Milivik", "vocab": 300, "width": 104, "norm": {"eps": 1e-5}, "embedding": {"scale": 9.0}, "logit_scale": 0.3,
         "layers": [{"type": "latent_attention", "mixer": latent, "mlp": {"kind": "dense", "ff": 136}},
                    {"type": "attention", "mixer": diff, "mlp": moe}, {"type": "latent_attention", "mixer": latent, "mlp": moe}]}
    d.update(over)
    return d
