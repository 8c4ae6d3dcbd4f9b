from .container import GepolixAttentionContainer, GepolixNonTransformerContainer, GepolixQueryContainer, GepolixStateSpaceContainer  # noqa: F401
from .model import GepolixInferenceModel, GepolixSpec  # noqa: F401
from .policy import GepolixPolicy  # noqa: F401
