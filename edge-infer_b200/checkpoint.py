"""Checkpoint admission for the verify path: HF-style decoder checkpoints (dense BF16 or AutoAWQ "GEMV" int4) to the
prepared-tensor names and layouts ei_model_create takes.

Mirrors what the reference does between a checkpoint and its prepared model:
  * AWQ metadata admission - only the 4-bit asymmetric GEMV packing, one agreed group size
    (bindings/python/include/decoder_weight_mapper.hpp:47-79, frontend/checkpoint.py:27-57);
  * tied / explicit output head (decoder_weight_mapper.hpp:81-102);
  * checkpoint key -> prepared name, kind and rank (decoder_weight_mapper.hpp:104-166, 219-253);
  * config.json -> decoder shape.
Linear weights stay in the checkpoint's own physical layout: [out, in] BF16, and for AWQ-GEMV
qweight int32 [out, in / 8], scales [out, groups (+ padding)], qzeros int32 [out, ceil(groups / 8)] - exactly what
the kernels stream, so nothing is repacked.

A minimal safetensors reader (the format is an 8-byte header length, a JSON header and raw little-endian data) is
included so that a local checkpoint directory can be read with numpy alone; nothing is ever fetched.
"""
from __future__ import annotations

import json
import re
import struct
from pathlib import Path
from typing import Dict, List, Mapping, Optional, Tuple

import numpy as np

from .runtime import (BLOCK_PARALLEL, MLP_RELU_SQUARED, Attention, ChannelDelta, LatentAttention, Layer, LayeredShape,
                      LinearAttention, PairEmbedding, Shape, StateSpace, Yarn)

DENSE, QWEIGHT, SCALES, ZEROS = 0, 1, 2, 3

MODEL_TYPES = ("qwen_bf16", "qwen_awq", "qwen3_bf16", "qwen3_awq", "zofesun_bf16", "zofesun_f32",
               "gikepel_bf16", "gikepel_f32")
_DESIGNS = {"Zofesun": "zofesun", "Gikepel": "gikepel"}  # `architecture` of layered designs

_PROJECTIONS = {
    "self_attn.q_proj": "wq", "self_attn.k_proj": "wk", "self_attn.v_proj": "wv", "self_attn.o_proj": "wo",
    "mlp.gate_proj": "w_gate", "mlp.up_proj": "w_up", "mlp.down_proj": "w_down",
}
_FORMATS = {"weight": DENSE, "qweight": QWEIGHT, "scales": SCALES, "qzeros": ZEROS}
_LAYER = re.compile(r"^model\.layers\.(0|[1-9][0-9]*)\.(.+)$")


def model_type_of(config: Mapping, dtype: str = "bfloat16") -> str:
    """The model type a config.json asks for: by `architecture` for designs that name themselves, by the Hugging Face
    `model_type` and quantization settings otherwise. dtype float32 is there for the layered designs only."""
    if dtype not in ("bfloat16", "float32"):
        raise ValueError("dtype must be bfloat16 or float32")
    design = _DESIGNS.get(config.get("architecture"))
    if design is not None:
        return design + ("_f32" if dtype == "float32" else "_bf16")
    family = {"qwen2": "qwen", "qwen3": "qwen3"}.get(config.get("model_type"))
    if family is None:
        raise ValueError("Unsupported model architecture: %r" % (config.get("architecture") or config.get("model_type")))
    if dtype != "bfloat16":
        raise NotImplementedError("This model family runs in bfloat16 only")
    return family + ("_awq" if "quantization_config" in config else "_bf16")


# ---------------------------------------------------------------- layered designs
def _size(section: Mapping, key: str, where: str, least: int = 1) -> int:
    value = section.get(key)
    if type(value) is not int or value < least:
        raise ValueError(f"{where}.{key} must be an integer of at least {least}")
    return value


def _number(section: Mapping, key: str, where: str) -> float:
    value = section.get(key)
    if isinstance(value, bool) or not isinstance(value, (int, float)):
        raise ValueError(f"{where}.{key} must be a number")
    return float(value)


def _section(parent: Mapping, key: str, where: str) -> Mapping:
    value = parent.get(key)
    if not isinstance(value, Mapping):
        raise ValueError(f"{where}.{key} must be an object")
    return value


def _zofesun_layer(entry: Mapping, where: str) -> Layer:
    mixer, layer = _section(entry, "mixer", where), Layer()
    kind = entry.get("type")
    if kind == "mingru":
        layer.rnn_width = _size(mixer, "width", where + ".mixer")
    elif kind == "parallel":
        left, right = _section(mixer, "left", where + ".mixer"), _section(mixer, "right", where + ".mixer")
        at = where + ".mixer.left"
        rot = _section(left, "rot", at)
        layer.attention = Attention(heads=_size(left, "heads", at), kv_heads=_size(left, "kv_heads", at),
                                    dim=_size(left, "dim", at), vdim=_size(left, "vdim", at),
                                    rot_dims=_size(rot, "dims", at + ".rot", 0), rot_base=_number(rot, "base", at + ".rot"),
                                    scale=_number(left, "scale", at))
        at = where + ".mixer.right"
        decay = right.get("decay")
        heads = _size(right, "heads", at)
        if not isinstance(decay, (list, tuple)) or len(decay) != heads:
            raise ValueError(at + ".decay must have one entry per head")
        layer.linear = LinearAttention(heads=heads, dim=_size(right, "dim", at), vdim=_size(right, "vdim", at),
                                       decay=[float(d) for d in decay])
        layer.left_scale = _number(mixer, "left_scale", where + ".mixer")
        layer.right_scale = _number(mixer, "right_scale", where + ".mixer")
    else:
        raise ValueError(f"{where}: unsupported mixer type {kind!r}")
    mlp = entry.get("mlp")
    if mlp is not None:
        if not isinstance(mlp, Mapping) or mlp.get("kind") != "dense":
            raise ValueError(where + ": unsupported feed-forward")
        layer.ff, layer.limit = _size(mlp, "ff", where + ".mlp"), _number(mlp, "limit", where + ".mlp")
    return layer


def _layer_entries(config: Mapping) -> List[Mapping]:
    entries = config.get("layers")
    if not isinstance(entries, list) or not entries or not all(isinstance(e, Mapping) for e in entries):
        raise ValueError("layers must be a nonempty list")
    return entries


def _layered_common(config: Mapping, true32: bool) -> Dict[str, object]:
    return dict(vocab_size=_size(config, "vocab", "config"), hidden_size=_size(config, "width", "config"),
                norm_eps=_number(_section(config, "norm", "config"), "eps", "norm"), true32=true32,
                max_position_embeddings=int(config.get("max_position_embeddings", 1 << 20)),
                bos_token_id=int(config.get("bos_token_id", 0) or 0),
                eos_token_id=_first_int(config.get("eos_token_id", 0xFFFFFFFF)))


def zofesun_shape(config: Mapping, true32: bool = False) -> LayeredShape:
    """Decoder shape of a Zofesun config.json: every size and constant comes from it."""
    entries = _layer_entries(config)
    loop = config.get("loop")
    if loop is not None:
        loop = (_size(loop, "start", "loop", 0), _size(loop, "stop", "loop"), _size(loop, "times", "loop"))
        if not loop[0] < loop[1] <= len(entries):
            raise ValueError("loop must span existing layers")
    return LayeredShape(layers=[_zofesun_layer(e, f"layers[{i}]") for i, e in enumerate(entries)], loop=loop,
                        **_layered_common(config, true32))


def _gikepel_layer(entry: Mapping, where: str) -> Layer:
    mixer, layer = _section(entry, "mixer", where), Layer(mlp=MLP_RELU_SQUARED)
    kind, at = entry.get("type"), where + ".mixer"
    if kind == "latent_attention":
        rot = _section(mixer, "rot", at)
        yarn = None
        if rot.get("scaling") is not None:
            scaling = _section(rot, "scaling", at + ".rot")
            yarn = Yarn(*(_number(scaling, key, at + ".rot.scaling") for key in ("factor", "original", "fast", "slow")))
        layer.latent = LatentAttention(*(_size(mixer, key, at) for key in ("heads", "dim", "rot_dim", "vdim", "kv_rank")),
                                       rot_dims=_size(rot, "dims", at + ".rot", 0), rot_base=_number(rot, "base", at + ".rot"),
                                       scale=_number(mixer, "scale", at), yarn=yarn)
    elif kind == "mamba2":
        layer.state_space = StateSpace(*(_size(mixer, key, at) for key in ("heads", "groups", "state", "vdim", "conv", "norm_groups")))
    elif kind == "channel_delta":
        layer.delta = ChannelDelta(*(_size(mixer, key, at) for key in ("heads", "kv_heads", "dim", "vdim", "conv")))
    else:
        raise ValueError(f"{where}: unsupported mixer type {kind!r}")
    mlp = entry.get("mlp")
    if mlp is not None:
        if not isinstance(mlp, Mapping) or mlp.get("kind") != "dense":
            raise ValueError(where + ": unsupported feed-forward")
        layer.ff = _size(mlp, "ff", where + ".mlp")
    return layer


def gikepel_shape(config: Mapping, true32: bool = False) -> LayeredShape:
    """Decoder shape of a Gikepel config.json. The ranks of the low-rank projections are not in it: they come from the
    checkpoint's tensors (with_ranks)."""
    pairs = config.get("embedding", {}).get("bigram")
    if pairs is not None:
        pairs = PairEmbedding(_size(pairs, "buckets", "embedding.bigram"), _size(pairs, "mul_prev", "embedding.bigram", 0),
                              _size(pairs, "mul_cur", "embedding.bigram", 0))
    softcap = 0.0 if config.get("logit_softcap") is None else _number(config, "logit_softcap", "config")
    return LayeredShape(layers=[_gikepel_layer(e, f"layers[{i}]") for i, e in enumerate(_layer_entries(config))],
                        block=BLOCK_PARALLEL, tied_embeddings=True, pairs=pairs, logit_softcap=softcap,
                        **_layered_common(config, true32))


def with_ranks(shape: LayeredShape, weights: Mapping) -> LayeredShape:
    """Fills in the ranks that only the tensors tell."""
    for i, layer in enumerate(shape.layers):
        if layer.delta is None:
            continue
        for name, field in (("a1", "decay_rank"), ("g1", "gate_rank")):
            tensor = weights.get(f"l{i}.mix.{name}")
            if tensor is None:
                raise ValueError(f"Decoder checkpoint lacks l{i}.mix.{name}")
            setattr(layer.delta, field, int(tensor.shape[0]))
    return shape


def layered_tensor_shapes(shape: LayeredShape) -> Dict[str, Tuple[int, ...]]:
    """Every tensor a layered checkpoint must hold, with its shape ([out, in] for linears, () for scalars)."""
    width, parallel = shape.hidden_size, shape.block == BLOCK_PARALLEL
    shapes: Dict[str, Tuple[int, ...]] = {"embed": (shape.vocab_size, width)}
    if not shape.tied_embeddings:
        shapes["head"] = (shape.vocab_size, width)
    if shape.pairs is not None:
        shapes["bigram"] = (shape.pairs.buckets + 1, width)

    def norm(name: str) -> None:
        shapes[name] = (width,)
        if not parallel:
            shapes.update({name + ".b": (width,), name + ".alpha": ()})

    norm("final.norm")
    if shape.loop is not None:
        shapes["loop.step"] = (shape.loop[2], width)
    for i, layer in enumerate(shape.layers):
        p = f"l{i}."
        norm(p + "norm1")
        if parallel:
            shapes[p + "ls1"] = (width,)
        else:
            norm(p + "norm1b")
        shapes.update({p + "mix." + name: dims for name, dims in _mixer_tensors(layer, width).items()})
        if layer.ff is not None:
            norm(p + "norm2")
            if parallel:
                shapes[p + "ls2"] = (width,)
            else:
                norm(p + "norm2b")
                shapes[p + "mlp.gate"] = (layer.ff, width)
            shapes.update({p + "mlp.up": (layer.ff, width), p + "mlp.down": (width, layer.ff)})
    return shapes


def _mixer_tensors(layer: Layer, width: int) -> Dict[str, Tuple[int, ...]]:
    if layer.rnn_width is not None:
        r = layer.rnn_width
        return {"z": (r, width), "z.b": (r,), "x": (r, width), "x.b": (r,), "g": (r, width), "o": (width, r)}
    if layer.latent is not None:
        a = layer.latent
        return {"q": (a.heads * (a.dim + a.rot_dim), width), "dkv": (a.kv_rank + a.rot_dim, width), "dkv.norm": (a.kv_rank,),
                "uk": (a.heads * a.dim, a.kv_rank), "uv": (a.heads * a.vdim, a.kv_rank), "g": (a.heads * a.vdim, width),
                "o": (width, a.heads * a.vdim)}
    if layer.state_space is not None:
        m = layer.state_space
        inner, pairs = m.heads * m.vdim, m.groups * m.state
        return {"in": (2 * inner + 2 * pairs + m.heads, width), "conv": (inner + 2 * pairs, m.taps),
                "conv.b": (inner + 2 * pairs,), "dt_bias": (m.heads,), "A_log": (m.heads,), "D": (m.heads,),
                "norm": (inner,), "o": (width, inner)}
    if layer.delta is not None:
        m = layer.delta
        keys, values = m.kv_heads * m.dim, m.heads * m.vdim
        return {"q": (keys, width), "q.conv": (keys, m.taps), "k": (keys, width), "k.conv": (keys, m.taps),
                "v": (values, width), "v.conv": (values, m.taps), "b": (m.heads, width), "A_log": (m.heads,),
                "norm": (m.vdim,), "a1": (m.decay_rank, width), "a2": (m.heads * m.dim, m.decay_rank),
                "dt_bias": (m.heads * m.dim,), "g1": (m.gate_rank, width), "g2": (values, m.gate_rank), "o": (width, values)}
    a, l = layer.attention, layer.linear
    return {"left.q": (a.heads * a.dim, width), "left.k": (a.kv_heads * a.dim, width), "left.v": (a.kv_heads * a.vdim, width),
            "left.sink": (a.heads,), "left.o": (width, a.heads * a.vdim), "right.q": (l.heads * l.dim, width),
            "right.k": (l.heads * l.dim, width), "right.v": (l.heads * l.vdim, width), "right.g": (l.heads * l.vdim, width),
            "right.o": (width, l.heads * l.vdim), "right.norm": (l.heads * l.vdim,)}


def _admit_layered(shape: LayeredShape, weights: Mapping):
    expected = layered_tensor_shapes(with_ranks(shape, weights))
    # Norms and scales of a feed-forward that a layer does not have, and the vectors of a loop that is not run, are
    # passed over.
    spare = {f"l{i}.{norm}{part}" for i, layer in enumerate(shape.layers) if layer.ff is None
             for norm in ("norm2", "norm2b", "ls2") for part in ("", ".b", ".alpha")} | {"loop.step"}
    missing, extra = sorted(set(expected) - set(weights)), sorted(set(weights) - set(expected) - spare)
    if missing:
        raise ValueError("Decoder checkpoint lacks " + missing[0])
    if extra:
        raise ValueError("Unsupported decoder weight key: " + extra[0])
    tensors: Dict[str, List[Tuple[int, object]]] = {}
    for name, dims in expected.items():
        payload = _bits(weights[name], name, DENSE)
        if tuple(int(d) for d in payload.shape) not in ((dims,) if dims else ((), (1,))):
            raise ValueError("Decoder checkpoint weight shape mismatch: " + name)
        tensors[name] = [(DENSE, payload)]
    return shape, tensors


def awq_group_size(config: Mapping) -> int:
    """Admits the AWQ metadata of a config (top level and `quantization_config`): the method must be AWQ, the
    packing GEMV, 4 bits, asymmetric, and every declared group size the same. Returns the group size (128 when
    none is declared)."""
    quantization = config.get("quantization_config", {})
    if not isinstance(quantization, Mapping):
        raise ValueError("quantization_config must be a dictionary")
    group: Optional[int] = None
    for settings in (config, quantization):
        method = settings.get("quant_method", "awq")
        if not isinstance(method, str) or method.lower() != "awq":
            raise ValueError("Only AWQ quant_method is supported")
        version = settings.get("version", "gemv")
        if not isinstance(version, str) or version.lower() != "gemv":
            raise ValueError("Only AWQ GEMV packing is supported")
        for key in ("bits", "w_bit"):
            if key in settings and (type(settings[key]) is not int or settings[key] != 4):
                raise ValueError("Only 4-bit AWQ packing is supported")
        if "zero_point" in settings and settings["zero_point"] is not True:
            raise ValueError("AWQ zero_point must be true for asymmetric packing")
        for key in ("group_size", "q_group_size"):
            if key not in settings:
                continue
            declared = settings[key]
            if type(declared) is not int or not 0 < declared <= 2**31 - 1:
                raise ValueError(f"AWQ {key} must be a positive integer")
            if group is not None and declared != group:
                raise ValueError("Contradictory AWQ group sizes")
            group = declared
    return 128 if group is None else group


def parse_name(source: str, qk_norm: bool, n_layers: int = 0) -> Tuple[str, int, int]:
    """Checkpoint key -> (prepared name, kind, rank). Raises ValueError for a key the decoder does not know, a
    malformed layer index or a layer beyond the configuration."""
    if source == "model.embed_tokens.weight":
        return "token_embeddings.weight", DENSE, 2
    if source == "model.norm.weight":
        return "rms_out_w", DENSE, 1
    for prefix in ("lm_head.", "model.lm_head."):
        if source.startswith(prefix):
            return _projection(source, "lm_head", "lm_head.bias", source[len(prefix):])
    match = _LAYER.match(source)
    if not match:
        if source.startswith("model.layers."):
            raise ValueError("Malformed decoder layer index: " + source)
        raise ValueError("Unsupported decoder weight key: " + source)
    layer, suffix = int(match.group(1)), match.group(2)
    if layer > 2**31 - 1:
        raise ValueError("Decoder layer index exceeds the supported range: " + source)
    if n_layers and layer >= n_layers:
        raise ValueError("Decoder weight layer exceeds configuration: " + source)
    norms = {"input_layernorm.weight": "rms_att_w", "post_attention_layernorm.weight": "rms_ffn_w"}
    if qk_norm:
        norms.update({"self_attn.q_norm.weight": "q_norm", "self_attn.k_norm.weight": "k_norm"})
    if suffix in norms:
        return f"{norms[suffix]}{layer}", DENSE, 1
    base, _, fmt = suffix.rpartition(".")
    if base in _PROJECTIONS:
        return _projection(source, f"{_PROJECTIONS[base]}{layer}", f"layers.{layer}.{base}.bias", fmt)
    raise ValueError("Unsupported decoder weight key: " + source)


def _projection(source: str, name: str, bias_name: str, fmt: str) -> Tuple[str, int, int]:
    if fmt == "bias":
        return bias_name, DENSE, 1
    if fmt in _FORMATS:
        return name, _FORMATS[fmt], 2
    raise ValueError("Unsupported decoder weight key: " + source)


def shape_from_config(config: Mapping, model_type: str):
    """Decoder shape from a config.json dictionary."""
    if model_type not in MODEL_TYPES:
        raise ValueError(f"Unsupported model type: {model_type}")
    if model_type.startswith("zofesun"):
        return zofesun_shape(config, true32=model_type.endswith("_f32"))
    if model_type.startswith("gikepel"):
        return gikepel_shape(config, true32=model_type.endswith("_f32"))
    heads = int(config["num_attention_heads"])
    head_dim = int(config.get("head_dim", int(config["hidden_size"]) // heads))
    awq = model_type.endswith("_awq")
    return Shape(vocab_size=int(config["vocab_size"]), n_layers=int(config["num_hidden_layers"]), n_heads=heads,
                 n_kv_heads=int(config.get("num_key_value_heads", heads)), hidden_size=int(config["hidden_size"]),
                 intermediate_size=int(config["intermediate_size"]), head_dim=head_dim,
                 max_position_embeddings=int(config.get("max_position_embeddings", 4096)),
                 rms_norm_eps=float(config.get("rms_norm_eps", 1e-6)), rope_theta=float(config.get("rope_theta", 1e6)),
                 quant_type=1 if awq else 0, group_size=awq_group_size(config) if awq else 128,
                 qk_norm=model_type.startswith("qwen3"), qkv_bias=not model_type.startswith("qwen3"),
                 tied_embeddings=False, bos_token_id=int(config.get("bos_token_id", 0) or 0),
                 eos_token_id=_first_int(config.get("eos_token_id", 0xFFFFFFFF)))


def _first_int(value) -> int:
    if isinstance(value, (list, tuple)):
        value = value[0]
    return int(value)


def _bits(array, name: str, kind: int):
    """Payload in the element type the library takes: BF16 as uint16 for dense / scales, int32 for packed data.
    Accepts numpy arrays and torch tensors (host or device); floating-point inputs are rounded to BF16."""
    if hasattr(array, "detach"):                             # torch tensor: stays where it is
        import torch
        if kind in (QWEIGHT, ZEROS):
            if array.dtype != torch.int32:
                raise ValueError("AWQ packed weights and zeros must have int32 dtype: " + name)
            return array.contiguous()
        return array.to(torch.bfloat16).contiguous()
    array = np.asarray(array)
    if kind in (QWEIGHT, ZEROS):
        if array.dtype.kind != "i" or array.dtype.itemsize != 4:
            raise ValueError("AWQ packed weights and zeros must have int32 dtype: " + name)
        return np.ascontiguousarray(array)
    if array.dtype == np.uint16:                             # already a BF16 payload
        return np.ascontiguousarray(array)
    from .synthetic import float_to_bf16
    return float_to_bf16(np.ascontiguousarray(array, dtype=np.float32))


def admit(config: Mapping, weights: Mapping, model_type: str):
    """(Shape, tensors for runtime.Model) from a config dictionary and a checkpoint's name -> array mapping.
    Validates names, ranks, AWQ completeness (packed weight, scales and zero points come together and never beside a
    dense weight of the same projection) and resolves a declared embedding tie."""
    shape = shape_from_config(config, model_type)
    if isinstance(shape, LayeredShape):
        return _admit_layered(shape, weights)
    tied = config.get("tie_word_embeddings", False)
    if not isinstance(tied, bool):
        raise ValueError("tie_word_embeddings must be a boolean")
    if "model.embed_tokens.weight" not in weights:
        raise ValueError("Decoder checkpoint requires model.embed_tokens.weight")
    has_head = any(key.startswith(("lm_head.", "model.lm_head.")) for key in weights)
    if not has_head and not tied:
        raise ValueError("Untied decoder checkpoint requires an explicit lm_head weight")
    tensors: Dict[str, List[Tuple[int, object]]] = {}
    for source, array in weights.items():
        if not isinstance(source, str):
            raise ValueError("Decoder checkpoint weight names must be strings")
        name, kind, rank = parse_name(source, shape.qk_norm, shape.n_layers)
        if kind != DENSE and shape.quant_type != 1:
            raise ValueError("Packed decoder weights require an AWQ model: " + name)
        payload = _bits(array, source, kind)
        if len(payload.shape) != rank:
            raise ValueError("Decoder checkpoint weight rank mismatch: " + name)
        entries = tensors.setdefault(name, [])
        if any(existing == kind for existing, _ in entries):
            raise ValueError("Duplicate normalized decoder weight: " + name)
        entries.append((kind, payload))
    for name, entries in tensors.items():
        kinds = {kind for kind, _ in entries}
        if kinds & {QWEIGHT, SCALES, ZEROS}:
            if DENSE in kinds:
                raise ValueError("Dense and AWQ weights overlap: " + name)
            if kinds != {QWEIGHT, SCALES, ZEROS}:
                raise ValueError("Incomplete AWQ decoder weight: " + name)
    shape.tied_embeddings = not has_head
    return shape, tensors


# ---------------------------------------------------------------- safetensors (read-only, numpy)
_DTYPES = {"BF16": (np.uint16, 2), "F16": (np.float16, 2), "F32": (np.float32, 4), "I32": (np.int32, 4),
           "I64": (np.int64, 8), "U8": (np.uint8, 1)}


def read_safetensors(path) -> Dict[str, np.ndarray]:
    """name -> array of one .safetensors file, memory-mapped. BF16 tensors come back as uint16 payloads."""
    path = Path(path)
    with path.open("rb") as handle:
        (header_bytes,) = struct.unpack("<Q", handle.read(8))
        header = json.loads(handle.read(header_bytes))
    data = np.memmap(path, dtype=np.uint8, mode="r", offset=8 + header_bytes)
    tensors = {}
    for name, entry in header.items():
        if name == "__metadata__":
            continue
        if entry["dtype"] not in _DTYPES:
            raise ValueError(f"Unsupported safetensors dtype {entry['dtype']}: {name}")
        dtype, _ = _DTYPES[entry["dtype"]]
        begin, end = entry["data_offsets"]
        tensors[name] = data[begin:end].view(dtype).reshape(entry["shape"])
    return tensors


def _checkpoint_file(root: Path, name) -> Path:
    if not isinstance(name, str) or not name or Path(name).is_absolute():
        raise ValueError("Checkpoint shard names must be relative paths")
    path = (root / name).resolve()
    if root not in path.parents:
        raise ValueError("Checkpoint shards must stay inside the model directory")
    if not path.is_file():
        raise FileNotFoundError(path)
    return path


def load_directory(model_path, model_type: Optional[str] = None):
    """(config, weights) of a local checkpoint directory: config.json plus model.safetensors or the shards its index
    names. Never fetches anything."""
    if model_type is not None and model_type not in MODEL_TYPES:
        raise ValueError(f"Unsupported model type: {model_type}")
    root = Path(model_path).resolve()
    config = json.loads((root / "config.json").read_text(encoding="utf-8"))
    if not isinstance(config, dict):
        raise ValueError("Model configuration must be a JSON object")
    index_path = root / "model.safetensors.index.json"
    if index_path.is_file():
        index = json.loads(index_path.read_text(encoding="utf-8"))
        weight_map = index.get("weight_map") if isinstance(index, dict) else None
        if not isinstance(weight_map, dict) or not weight_map:
            raise ValueError("The safetensors index must contain a nonempty weight_map")
        shards = sorted({_checkpoint_file(root, shard) for shard in weight_map.values()})
        wanted = set(weight_map)
    else:
        shards, wanted = [_checkpoint_file(root, "model.safetensors")], None
    weights: Dict[str, np.ndarray] = {}
    for shard in shards:
        for name, array in read_safetensors(shard).items():
            if wanted is None or name in wanted:
                weights[name] = array
    if not weights:
        raise ValueError("The checkpoint contains no tensors")
    return config, weights
