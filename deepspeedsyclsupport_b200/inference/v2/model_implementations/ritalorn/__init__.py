from .container import RitalornAttentionContainer, RitalornLatentContainer, RitalornNonTransformerContainer, RitalornQueryContainer  # noqa: F401
from .model import RitalornInferenceModel, RitalornSpec  # noqa: F401
from .policy import RitalornPolicy  # noqa: F401
