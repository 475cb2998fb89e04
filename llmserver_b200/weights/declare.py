"""What tensors a model needs: collected from the parts its specification names."""
from __future__ import annotations

from dataclasses import dataclass
from typing import Dict, Tuple

MATRIX = "matrix"   # random mode: N(0, 0.02)
NORM = "norm"       # random mode: 1 + N(0, 0.1)
OFFSET = "offset"   # a norm weight stored as its distance from one; random mode: N(0, 0.1)
TABLE = "table"     # integer table (kept as int32)
WIDE = "wide"       # always held in float32, whatever the compute dtype (routers, per-head scalars); random mode: N(0, 0.02)
MIXING = "mixing"   # coefficients between residual streams, held in float32 as WIDE; random mode: N(0, 0.1) around the identity (a
                    # matrix) or around one (a vector), so that the streams stay of their size


@dataclass(frozen=True)
class WeightDecl:
    shape: Tuple[int, ...]
    kind: str = MATRIX


def declared_weights(spec) -> Dict[str, WeightDecl]:
    """Full tensor name -> declaration, for every tensor the model reads from a checkpoint."""
    from ..parts import registry as parts

    wanted: Dict[str, WeightDecl] = {spec.embedding_name: WeightDecl((spec.vocab_size, spec.hidden_size))}
    for layer in spec.layers:
        # what the block arrangement itself reads (scales on its sub-layers' outputs, say) lies behind the layer's prefix
        for local, declaration in parts.BLOCKS.get(layer.block.kind).declare_weights(layer.block.as_dict()).items():
            wanted[layer.prefix + local] = declaration
        for _, part_spec, part_cls, prefix in parts.parts_of_layer(layer):
            for local, declaration in part_cls.declare_weights(part_spec.as_dict()).items():
                wanted[prefix + local] = declaration
    for local, declaration in parts.NORMS.get(spec.final_norm.kind).declare_weights(spec.final_norm.as_dict()).items():
        wanted[spec.final_norm_prefix + local] = declaration
    for name, position in spec.positions.items():
        for local, declaration in parts.POSITION_ENCODINGS.get(position.kind).declare_weights(position.as_dict()).items():
            wanted[f"model.positions.{name}.{local}"] = declaration
    if not spec.tie_head:
        wanted[spec.head_name] = WeightDecl((spec.vocab_size, spec.hidden_size))
    return wanted
