"""Model families: ``config.json`` -> this engine's model configuration, and model directories -> loaded models.

Two Hugging Face decoder families (``model_type``) become a ``LlamaConfig``, both pre-norm transformers with RMSNorm, rotary embeddings,
SwiGLU and (grouped-query) attention with head_dim 128:

  llama   Llama 2 / 3 (``model_type: llama``); optional llama3 rope scaling (low_freq_factor 1,
          high_freq_factor 4, original context 8192 are the only accepted parameters); optional tied
          embeddings
  qwen3   Qwen3 dense models (``model_type: qwen3``): as llama plus per-head RMSNorm on queries and keys

A file that names an ``architecture`` instead lists its layers one by one:

  Dulisun  chunked attention with a sink, mixtures of experts, output norms (``models/dulisun.py``); served only
  Zafopel  latent attention beside the feed-forward, mixtures with scaled inputs, elementwise norms (``models/zafopel.py``); served only

Anything the kernels do not implement is rejected here with a clear message (linear biases, attention
dropout, other rope scaling types, head_dim != 128, sliding windows). Reference:
RPEG/runtime/models/base.py:19-58, llama.py:17-79, qwen3.py:17-60, registry.py:23-52.
"""
from __future__ import annotations

import json
from pathlib import Path
from typing import Any, Callable, Dict, List, Mapping, NamedTuple, Union

from ..ops.kernels import LATENT_MAX_RANK
from ..runtime.errors import RuntimeConfigError
from .dulisun import AttentionMixer, DecoderLayer, DulisunConfig, DulisunModel, ExpertMixture
from .llama import LlamaConfig, LlamaModel
from .zafopel import DenseFF, InputScaledMixture, LatentMixer, ParallelLayer, ZafopelConfig, ZafopelModel

FAMILIES = ("llama", "qwen3")
ServedConfig = Union[DulisunConfig, ZafopelConfig]


def _llama3_rope_factor(cfg: Mapping[str, Any]) -> float:
    raw = cfg.get("rope_scaling")
    if raw is None:
        return 1.0
    if not isinstance(raw, Mapping):
        raise RuntimeConfigError("rope_scaling must be a JSON object when provided")
    kind = raw.get("rope_type", raw.get("type"))
    if kind in (None, "default"):
        return 1.0
    if kind != "llama3":
        raise RuntimeConfigError(f"unsupported rope_scaling type {kind!r}; only llama3 scaling is implemented")
    if float(raw.get("low_freq_factor", 1.0)) != 1.0 or float(raw.get("high_freq_factor", 4.0)) != 4.0 \
            or int(raw.get("original_max_position_embeddings", 8192)) != 8192:
        raise RuntimeConfigError("unsupported llama3 rope_scaling factors (need low_freq_factor=1, high_freq_factor=4, "
                                 "original_max_position_embeddings=8192)")
    return max(1.0, float(raw.get("factor", 1.0)))


def _attention_mixer(m: Mapping[str, Any], where: str) -> AttentionMixer:
    heads, kv, dim = int(m["heads"]), int(m["kv_heads"]), int(m["dim"])
    rot = m.get("rot") or {}
    rot_dims = int(rot.get("dims", 0))
    mask = m.get("mask") or {}
    if heads < 1 or kv < 1 or heads % kv:
        raise RuntimeConfigError(f"{where}: {heads} query heads do not divide over {kv} key/value heads")
    if int(m.get("vdim", dim)) != dim:
        raise RuntimeConfigError(f"{where}: the values are the projected keys, so vdim must equal dim ({dim}), got {m['vdim']}")
    if not 1 <= dim <= 256:
        raise RuntimeConfigError(f"{where}: head size {dim} is not supported (the attention kernels cover 1 to 256)")
    if rot_dims < 0 or rot_dims > dim or rot_dims % 2:
        raise RuntimeConfigError(f"{where}: rot.dims must be even and at most dim, got {rot_dims}")
    window = int(mask.get("size", 0))
    if mask and window < 1:
        raise RuntimeConfigError(f"{where}: mask.size must be at least 1")
    return AttentionMixer(heads=heads, kv_heads=kv, dim=dim, scale=float(m["scale"]), window=window, rot_dims=rot_dims,
                          rot_base=float(rot.get("base", 10000.0)))


def _expert_mixture(m: Mapping[str, Any], where: str) -> ExpertMixture:
    if m.get("kind", "moe") != "moe":
        raise RuntimeConfigError(f"{where}: unsupported feed-forward kind {m['kind']!r}; only moe is implemented")
    r = m["router"]
    groups = r.get("groups") or {"count": 1, "keep": 1}
    shared = m.get("shared") or {}
    e = ExpertMixture(experts=int(r["experts"]), top=int(r["top"]), ff=int(m["expert"]["ff"]), shared_ff=int(shared.get("ff", 0)),
                      groups=int(groups["count"]), keep=int(groups["keep"]))
    if e.experts < 1 or e.ff < 1 or e.groups < 1 or e.experts % e.groups or not 1 <= e.keep <= e.groups:
        raise RuntimeConfigError(f"{where}: {e.experts} experts do not form {e.groups} equal groups of which {e.keep} are kept")
    if not 1 <= e.top <= e.keep * (e.experts // e.groups):
        raise RuntimeConfigError(f"{where}: cannot choose {e.top} experts from {e.keep} groups of {e.experts // e.groups}")
    if e.segments > 1024:
        raise RuntimeConfigError(f"{where}: {e.segments} expert segments exceed the kernels' limit of 1024")
    return e


def dulisun_config(cfg: Mapping[str, Any], max_pos: int | None = None) -> DulisunConfig:
    layers = []
    for i, l in enumerate(cfg["layers"]):
        if l.get("type") != "attention":
            raise RuntimeConfigError(f"layer {i}: unsupported mixer type {l.get('type')!r}; only attention is implemented")
        mlp = l.get("mlp")
        layers.append(DecoderLayer(_attention_mixer(l["mixer"], f"layer {i} mixer"),
                                   None if mlp is None else _expert_mixture(mlp, f"layer {i} mlp")))
    if not layers:
        raise RuntimeConfigError("the model has no layers")
    return DulisunConfig(width=int(cfg["width"]), vocab=int(cfg["vocab"]), layers=tuple(layers), norm_eps=float(cfg["norm"]["eps"]),
                         max_pos=int(max_pos or 4096))


def dulisun_config_dict(cfg: DulisunConfig) -> Dict[str, Any]:
    """The inverse of ``dulisun_config``."""
    layers = []
    for l in cfg.layers:
        m, e = l.mixer, l.mlp
        mixer: Dict[str, Any] = {"heads": m.heads, "kv_heads": m.kv_heads, "dim": m.dim, "vdim": m.dim, "scale": m.scale}
        if m.window:
            mixer["mask"] = {"size": m.window}
        if m.rot_dims:
            mixer["rot"] = {"base": m.rot_base, "dims": m.rot_dims}
        mlp: Dict[str, Any] | None = None
        if e is not None:
            mlp = {"kind": "moe", "expert": {"ff": e.ff}, "router": {"experts": e.experts, "top": e.top, "groups": {"count": e.groups, "keep": e.keep}}}
            if e.shared_ff:
                mlp["shared"] = {"ff": e.shared_ff}
        layers.append({"type": "attention", "mixer": mixer, "mlp": mlp})
    return {"architecture": "Dulisun", "vocab": cfg.vocab, "width": cfg.width, "norm": {"eps": cfg.norm_eps}, "layers": layers}


def _latent_mixer(kind: str, m: Mapping[str, Any], where: str, index: int, before: List[ParallelLayer]) -> LatentMixer:
    """``latent_attention``: queries straight from the input, sliding window. ``latent_attention_2``: queries through a latent of their own,
    causal, with a sink."""
    second = kind == "latent_attention_2"
    heads, dim, rot_dim, vdim, rank = (int(m[k]) for k in ("heads", "dim", "rot_dim", "vdim", "kv_rank"))
    rot = m["rot"]
    if min(heads, dim, vdim, rank) < 1:
        raise RuntimeConfigError(f"{where}: heads, dim, vdim and kv_rank must be at least 1")
    if rot_dim < 0 or rot_dim % 2 or int(rot.get("dims", rot_dim)) != rot_dim:
        raise RuntimeConfigError(f"{where}: the rotated part is rotated as a whole, so rot.dims must equal rot_dim and be even, got {rot.get('dims')}, {rot_dim}")
    if rank > LATENT_MAX_RANK:
        raise RuntimeConfigError(f"{where}: kv_rank {rank} is not supported (the attention kernels cover up to {LATENT_MAX_RANK})")
    q_rank = int(m["q_rank"]) if second else 0
    if second and not 1 <= q_rank <= 8192:
        raise RuntimeConfigError(f"{where}: q_rank must lie in 1 to 8192, got {q_rank}")
    mask = m.get("mask") or {}
    window = int(mask.get("size", 0))
    if mask and (second or window < 1):
        raise RuntimeConfigError(f"{where}: " + ("this mixer is causal and takes no mask" if second else "mask.size must be at least 1"))
    src = m.get("kv_from")
    out = LatentMixer(heads=heads, dim=dim, rot_dim=rot_dim, vdim=vdim, kv_rank=rank, scale=float(m["scale"]), rot_base=float(rot["base"]),
                      q_rank=q_rank, window=window, sink=second, kv_from=None if src is None else int(src))
    if src is not None:
        j = int(src)
        if not 0 <= j < index or before[j].mixer.kv_from is not None:
            raise RuntimeConfigError(f"{where}: kv_from must name an earlier layer with a latent of its own, got {j}")
        o = before[j].mixer
        if (o.kv_rank, o.rot_dim, o.rot_base) != (rank, rot_dim, out.rot_base):
            raise RuntimeConfigError(f"{where}: kv_rank, rot_dim and rotation must equal those of layer {j}, whose latents it reads")
    return out


def _parallel_ff(m: Mapping[str, Any], where: str) -> DenseFF | InputScaledMixture:
    kind = m.get("kind")
    if kind == "dense":
        if int(m["ff"]) < 1:
            raise RuntimeConfigError(f"{where}: ff must be at least 1")
        return DenseFF(int(m["ff"]))
    if kind != "moe":
        raise RuntimeConfigError(f"{where}: unsupported feed-forward kind {kind!r}; dense and moe are implemented")
    e = InputScaledMixture(experts=int(m["router"]["experts"]), top=int(m["router"]["top"]), ff=int(m["expert"]["ff"]))
    if e.ff < 1 or not 1 <= e.top <= e.experts:
        raise RuntimeConfigError(f"{where}: cannot choose {e.top} of {e.experts} experts of size {e.ff}")
    if e.experts > 1024:
        raise RuntimeConfigError(f"{where}: {e.experts} experts exceed the kernels' limit of 1024")
    return e


def zafopel_config(cfg: Mapping[str, Any], max_pos: int | None = None) -> ZafopelConfig:
    layers: List[ParallelLayer] = []
    for i, l in enumerate(cfg["layers"]):
        if l.get("type") not in ("latent_attention", "latent_attention_2"):
            raise RuntimeConfigError(f"layer {i}: unsupported mixer type {l.get('type')!r}; latent_attention and latent_attention_2 are implemented")
        mlp = l.get("mlp")
        layers.append(ParallelLayer(_latent_mixer(l["type"], l["mixer"], f"layer {i} mixer", i, layers),
                                    None if mlp is None else _parallel_ff(mlp, f"layer {i} mlp")))
    if not layers:
        raise RuntimeConfigError("the model has no layers")
    return ZafopelConfig(width=int(cfg["width"]), vocab=int(cfg["vocab"]), layers=tuple(layers), norm_eps=float(cfg["norm"]["eps"]),
                         max_pos=int(max_pos or 4096))


def zafopel_config_dict(cfg: ZafopelConfig) -> Dict[str, Any]:
    """The inverse of ``zafopel_config``."""
    layers = []
    for l in cfg.layers:
        m, e = l.mixer, l.mlp
        mixer: Dict[str, Any] = {"heads": m.heads, "dim": m.dim, "rot_dim": m.rot_dim, "vdim": m.vdim, "kv_rank": m.kv_rank, "scale": m.scale,
                                 "rot": {"base": m.rot_base, "dims": m.rot_dim}}
        if m.q_rank:
            mixer["q_rank"] = m.q_rank
        if m.window:
            mixer["mask"] = {"size": m.window}
        if m.kv_from is not None:
            mixer["kv_from"] = m.kv_from
        mlp: Dict[str, Any] | None = None
        if isinstance(e, DenseFF):
            mlp = {"kind": "dense", "ff": e.ff}
        elif e is not None:
            mlp = {"kind": "moe", "expert": {"ff": e.ff}, "router": {"experts": e.experts, "top": e.top}}
        layers.append({"type": "latent_attention_2" if m.sink else "latent_attention", "mixer": mixer, "mlp": mlp})
    return {"architecture": "Zafopel", "vocab": cfg.vocab, "width": cfg.width, "norm": {"eps": cfg.norm_eps}, "layers": layers}


class _Architecture(NamedTuple):
    config: type
    model: type
    read: Callable[..., ServedConfig]
    write: Callable[[Any], Dict[str, Any]]


ARCHITECTURES: Dict[str, _Architecture] = {
    "Dulisun": _Architecture(DulisunConfig, DulisunModel, dulisun_config, dulisun_config_dict),
    "Zafopel": _Architecture(ZafopelConfig, ZafopelModel, zafopel_config, zafopel_config_dict),
}


def _architecture_of(cfg) -> _Architecture | None:
    return next((a for a in ARCHITECTURES.values() if isinstance(cfg, a.config)), None)


def config_from_hf(hf: Mapping[str, Any], *, max_pos: int | None = None, lm_head: bool = True, scalar_head: bool = False) -> LlamaConfig | ServedConfig:
    if "architecture" in hf:
        if hf["architecture"] not in ARCHITECTURES:
            raise RuntimeConfigError(f"unsupported architecture {hf['architecture']!r}; supported: {', '.join(ARCHITECTURES)}")
        if scalar_head or not lm_head:
            raise RuntimeConfigError(f"{hf['architecture']} models have a language-model head only")
        return ARCHITECTURES[hf["architecture"]].read(hf, max_pos)
    family = hf.get("model_type")
    if family not in FAMILIES:
        raise RuntimeConfigError(f"unsupported model_type {family!r}; supported: {', '.join(FAMILIES)}")
    hidden, heads = int(hf["hidden_size"]), int(hf["num_attention_heads"])
    head_dim = int(hf.get("head_dim") or hidden // heads)
    if head_dim != 128:
        raise RuntimeConfigError(f"head_dim {head_dim} is not supported (the attention kernels are built for 128)")
    if hf.get("attention_bias") or hf.get("mlp_bias"):
        raise RuntimeConfigError("linear biases are not supported")
    if float(hf.get("attention_dropout", 0.0)) != 0.0:
        raise RuntimeConfigError("attention dropout is not supported")
    if hf.get("use_sliding_window") or (hf.get("sliding_window") and family != "qwen3"):
        raise RuntimeConfigError("sliding-window attention is not supported")
    if str(hf.get("hidden_act", "silu")) != "silu":
        raise RuntimeConfigError("only the SiLU-gated MLP is supported")
    return LlamaConfig(
        n_layers=int(hf["num_hidden_layers"]), d_model=hidden, d_ff=int(hf["intermediate_size"]), n_heads=heads,
        n_kv_heads=int(hf.get("num_key_value_heads", heads)), head_dim=head_dim, vocab=int(hf["vocab_size"]),
        rms_eps=float(hf.get("rms_norm_eps", 1e-6 if family == "qwen3" else 1e-5)),
        rope_theta=float(hf.get("rope_theta", 1e6 if family == "qwen3" else 5e5)),
        max_pos=int(max_pos or min(int(hf.get("max_position_embeddings", 8192)), 32768)),
        lm_head=lm_head, scalar_head=scalar_head, qk_norm=family == "qwen3",
        tie_embeddings=bool(hf.get("tie_word_embeddings", False)),
        rope_scaling_factor=_llama3_rope_factor(hf) if family == "llama" else 1.0, family=family)


def config_from_hf_path(path, **kw) -> LlamaConfig | ServedConfig:
    p = Path(path)
    cfg_file = p / "config.json" if p.is_dir() else p
    if not cfg_file.exists():
        raise RuntimeConfigError(f"{cfg_file} does not exist")
    return config_from_hf(json.loads(cfg_file.read_text()), **kw)


def model_class(cfg):
    """The model class that runs a configuration."""
    arch = _architecture_of(cfg)
    return LlamaModel if arch is None else arch.model


def load_model(path, device, *, dtype=None, max_pos: int | None = None):
    """Build the model a directory describes (``config.json`` chooses the class) and load its weights. ``dtype``: bfloat16
    (default) or, for families that run in it, float32. Compiles the family's kernels if they are not built yet."""
    import torch

    from ..ops import _lib
    from ..runtime.hf import load_weights
    cfg = config_from_hf_path(path, max_pos=max_pos)
    cls = model_class(cfg)
    dtype = dtype or torch.bfloat16
    if cls is LlamaModel and dtype != torch.bfloat16:
        raise RuntimeConfigError(f"{cfg.family} models run in bfloat16 only")
    if torch.device(device).type == "cuda":
        _lib.ensure(cls.KERNEL_SOURCES)
    model = cls(cfg, device) if cls is LlamaModel else cls(cfg, device, dtype=dtype, seed=None)
    load_weights(model, path)
    return model


def hf_config_dict(cfg) -> Dict[str, Any]:
    """The inverse mapping (used when exporting a checkpoint next to its architecture)."""
    arch = _architecture_of(cfg)
    if arch is not None:
        return arch.write(cfg)
    out: Dict[str, Any] = {
        "model_type": cfg.family, "hidden_size": cfg.d_model, "intermediate_size": cfg.d_ff, "num_hidden_layers": cfg.n_layers,
        "num_attention_heads": cfg.n_heads, "num_key_value_heads": cfg.n_kv_heads, "head_dim": cfg.head_dim, "vocab_size": cfg.vocab,
        "rms_norm_eps": cfg.rms_eps, "rope_theta": cfg.rope_theta, "max_position_embeddings": cfg.max_pos, "hidden_act": "silu",
        "tie_word_embeddings": cfg.tie_embeddings, "attention_bias": False, "torch_dtype": "bfloat16"}
    if cfg.rope_scaling_factor > 1.0:
        out["rope_scaling"] = {"rope_type": "llama3", "factor": cfg.rope_scaling_factor, "low_freq_factor": 1.0, "high_freq_factor": 4.0,
                               "original_max_position_embeddings": 8192}
    return out
